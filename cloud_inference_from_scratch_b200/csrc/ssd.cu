// State-space recurrence with ONE decay per head and token (Mamba-2's state-space duality):
//
//     dt_t = softplus(r_t + bias_h)                          (r: the projection's rate column of head h)
//     S_t  = exp(-exp(A_h) * dt_t) S_(t-1) + dt_t * B_t x_t^T      S: [state][vdim], float32, per request and head
//     y_t  = S_t^T C_t + D_h x_t
//
// Heads come in equal groups of neighbours that share B and C.  x, B and C arrive as float32 rows (after their short
// convolution), the rate as a column of the projection.  Everything is float32.
//
// Single tokens (and any batch): `ssd_scan_kernel` walks the tokens with the state in registers.
//
// Prompt portions run in chunks of kChunk tokens.  With b_t = sum of the log decays from the chunk's first token to
// t (all exponents below are <= 0):
//   1. per (chunk, head)         dt_t and b_t, and what the whole chunk leaves of a state
//   2. per (chunk, group)        G_ij = C_i . B_j for j <= i (shared by the group's heads)
//   3. per (chunk, head)         U = sum_j exp(b_last - b_j) dt_j B_j x_j^T
//   4. per (request, head)       walks its chunks, S <- exp(b_last) S + U, leaving the state BEFORE the chunk in U's
//                                place; the last S goes to the slot
//   5. per (chunk, head)         y_i = exp(b_i) S_before^T C_i + sum_(j<=i) exp(b_i - b_j) dt_j G_ij x_j + D x_i
// Products 2, 3 and 5 are 64 x 64 tiles, four by four numbers a thread; for 16-bit runs 3 and 5 run on the tensor cores
// (see there).  2 rides in the launch of 3.  A request's result depends on its own tokens
// and state only, whatever the batch or the slot, and on the cut of its prompt only through the order of additions.
#include "common.cuh"

CIE_DEFINE_LAST_ERROR()

namespace cie {

constexpr int kWarps = 8;
constexpr int kMaxState = 256;
constexpr int kChunk = 64;
constexpr int kTile = 64;
constexpr int kLd = kTile + 4;       // padded tile row: 16-byte pieces, few bank conflicts

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <int V> __device__ __forceinline__ void load_v(float (&dst)[V], const float* src) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(src);
    dst[0] = v.x; dst[1] = v.y; dst[2] = v.z; dst[3] = v.w;
  } else {
    dst[0] = src[0];
  }
}
template <int V> __device__ __forceinline__ void store_v(float* dst, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
  else dst[0] = v[0];
}

// Columns of a float32 row: x (heads x vdim), B and C (groups x state) of `rows`; the rate of `proj`.
struct Inputs {
  const float* rows;
  int stride, x_off, b_off, c_off;
  const float* proj;
  int proj_stride, r_off;
  const float* a_log;
  const float* dt_bias;
  const float* skip;       // D
  int heads, groups, state, vdim;
};

// ---------------------------------------------------------------- token by token
// grid (requests, heads, ceil(vdim / 32)); warp w owns the state rows w, w + 8, ..., lane = value column.
template <int R>
__global__ void __launch_bounds__(kWarps * 32)
ssd_scan_kernel(Inputs in, float* __restrict__ out, int out_stride, float* __restrict__ state, long long state_stride,
                const int* __restrict__ query_start, const int* __restrict__ slots,
                const int* __restrict__ request_active, int max_slots, int* err) {
  __shared__ float b_s[2][kWarps * R], c_s[2][kWarps * R];
  __shared__ float part_s[2][kWarps][32];
  pdl_wait();
  pdl_trigger();
  const int request = blockIdx.x, head = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int column = blockIdx.z * 32 + lane, n = in.state;
  const bool live = column < in.vdim;
  const int slot = slots[request];
  if (slot < 0 || slot >= max_slots) {
    if (threadIdx.x == 0) atomicOr(err, kErrBadRequest);
    return;
  }
  const int begin = query_start[request], end = query_start[request + 1];
  const int group = head / (in.heads / in.groups);
  const float rate = -expf(in.a_log[head]), bias = in.dt_bias[head], skip = in.skip[head];
  float* s_base = state + (size_t)slot * state_stride + (size_t)head * n * in.vdim;
  float s[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = warp + kWarps * r;
    s[r] = (i < n && live) ? s_base[(size_t)i * in.vdim + column] : 0.f;
  }
  for (int t = begin; t < end; ++t) {
    const int buf = (t - begin) & 1;
    const float* row = in.rows + (size_t)t * in.stride;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      b_s[buf][i] = row[in.b_off + group * n + i];
      c_s[buf][i] = row[in.c_off + group * n + i];
    }
    const float x = live ? row[in.x_off + head * in.vdim + column] : 0.f;
    const float dt = softplus_f(in.proj[(size_t)t * in.proj_stride + in.r_off + head] + bias);
    const float keep = expf(rate * dt), gained = dt * x;
    __syncthreads();
    float o = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = warp + kWarps * r;
      if (i < n) {
        s[r] = fmaf(keep, s[r], b_s[buf][i] * gained);
        o = fmaf(s[r], c_s[buf][i], o);
      }
    }
    part_s[buf][warp][lane] = o;
    __syncthreads();
    if (warp == 0 && live) {
      float total = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) total += part_s[buf][w][lane];
      out[(size_t)t * out_stride + head * in.vdim + column] = fmaf(skip, x, total);
    }
    // the buffers of token t are written again only after the first barrier of token t + 2
  }
  if (request_active[request] && live) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = warp + kWarps * r;
      if (i < n) s_base[(size_t)i * in.vdim + column] = s[r];
    }
  }
}

// ---------------------------------------------------------------- chunks
// grid (chunks, ceil(heads / 32)): the rates of 32 heads side by side in shared memory; a warp sums four heads over
// the chunk's tokens, two tokens a lane.  gates: [T][heads] of (dt, b as two floats, 0); decays: [chunks][heads], exp of the
// chunk's last b.  b can be large beside the difference of two of them that an exponential takes, so it is summed in
// double and kept as a float and what that leaves over.
__global__ void __launch_bounds__(256)
ssd_gates_kernel(Inputs in, float4* __restrict__ gates, float* __restrict__ decays, const int* __restrict__ chunk_row,
                 const int* __restrict__ chunk_count) {
  static_assert(kChunk == 64, "two tokens a lane");
  __shared__ float dt_s[kChunk][33];
  __shared__ double sum_s[kChunk][33];
  pdl_wait();
  pdl_trigger();
  const int head0 = blockIdx.y * 32, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row0 = chunk_row[blockIdx.x], n = chunk_count[blockIdx.x];
  const bool mine = head0 + lane < in.heads;
  const float bias = mine ? in.dt_bias[head0 + lane] : 0.f, rate = mine ? -expf(in.a_log[head0 + lane]) : 0.f;
#pragma unroll
  for (int u = 0; u < kChunk / kWarps; ++u) {
    const int j = warp + kWarps * u;
    float d = 0.f;
    if (mine && j < n) d = softplus_f(in.proj[(size_t)(row0 + j) * in.proj_stride + in.r_off + head0 + lane] + bias);
    dt_s[j][lane] = d;
    sum_s[j][lane] = (double)(rate * d);
  }
  __syncthreads();
#pragma unroll
  for (int h = warp * 4; h < warp * 4 + 4; ++h) {
    double first = sum_s[2 * lane][h];
    double second = first + sum_s[2 * lane + 1][h];
    double before = second;               // the sum over this lane's tokens and all earlier ones
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
      const double other = __shfl_up_sync(0xffffffffu, before, offset);
      if (lane >= offset) before += other;
    }
    before = __shfl_up_sync(0xffffffffu, before, 1);
    if (lane == 0) before = 0.0;
    sum_s[2 * lane][h] = before + first;
    sum_s[2 * lane + 1][h] = before + second;
  }
  __syncthreads();
  if (!mine) return;
#pragma unroll
  for (int u = 0; u < kChunk / kWarps; ++u) {
    const int j = warp + kWarps * u;
    const float b = (float)sum_s[j][lane];
    if (j < n) gates[(size_t)(row0 + j) * in.heads + head0 + lane] = make_float4(dt_s[j][lane], b, (float)(sum_s[j][lane] - b), 0.f);
    if (j == n - 1) decays[(size_t)blockIdx.x * in.heads + head0 + lane] = expf(b);
  }
}

// acc[a][b] += sum over `depth` rows of left[k][4 ty + a] * right[k][4 tx + b]
__device__ __forceinline__ void tile_product(float (&acc)[4][4], const float* left, const float* right, int depth, int ty, int tx) {
#pragma unroll 4
  for (int k = 0; k < depth; ++k) {
    const float4 l = *reinterpret_cast<const float4*>(left + k * kLd + 4 * ty);
    const float4 r = *reinterpret_cast<const float4*>(right + k * kLd + 4 * tx);
    const float lv[4] = {l.x, l.y, l.z, l.w}, rv[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
      for (int b = 0; b < 4; ++b) acc[a][b] = fmaf(lv[a], rv[b], acc[a][b]);
  }
}

// dst[j][c] = src[(row0 + j)][col + c] * factor(j) for j < 64, c < 64; zero outside n rows and `width` columns.
template <typename F>
__device__ __forceinline__ void stage_rows(float* dst, const float* src, int stride, int row0, int n, int col, int width, F factor) {
  if (((reinterpret_cast<uintptr_t>(src + (size_t)row0 * stride + col) & 15) == 0) && stride % 4 == 0 && width % 4 == 0) {
#pragma unroll
    for (int e = threadIdx.x; e < kTile * (kTile / 4); e += 256) {
      const int j = e / (kTile / 4), c = (e % (kTile / 4)) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (j < n && c < width) v = *reinterpret_cast<const float4*>(src + (size_t)(row0 + j) * stride + col + c);
      const float f = factor(j);
      *reinterpret_cast<float4*>(dst + j * kLd + c) = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
    }
    return;
  }
  for (int e = threadIdx.x; e < kTile * kTile; e += 256) {
    const int j = e / kTile, c = e % kTile;
    dst[j * kLd + c] = (j < n && c < width) ? src[(size_t)(row0 + j) * stride + col + c] * factor(j) : 0.f;
  }
}

// dst[c][j] = src[(row0 + j)][col + c]: the same tile with tokens along the fast axis.  A thread takes one token's
// piece of four columns; neighbouring threads take neighbouring tokens, so that the stores do not collide.
__device__ __forceinline__ void stage_columns(float* dst, const float* src, int stride, int row0, int n, int col, int width) {
  const bool wide = ((reinterpret_cast<uintptr_t>(src + (size_t)row0 * stride + col) & 15) == 0) && stride % 4 == 0 && width % 4 == 0;
  for (int e = threadIdx.x; e < kTile * (kTile / 4); e += 256) {
    const int j = e % kTile, c = (e / kTile) * 4;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (j < n) {
      const float* s = src + (size_t)(row0 + j) * stride + col + c;
      if (wide && c < width) {
        const float4 q = *reinterpret_cast<const float4*>(s);
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
      } else {
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (c + x < width) v[x] = s[x];
      }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) dst[(c + x) * kLd + j] = v[x];
  }
}

// G of a (chunk, group): products[chunk][group][j][i] = C_i . B_j, or, `by_query`, [i][j]: the row that step 5 reads
// together.  tiles: shared memory for two tiles.
__device__ __forceinline__ void chunk_products(const Inputs& in, float* products, int chunk, int group, int row0, int n,
                                               bool by_query, float* tiles) {
  float *b_s = tiles, *c_s = tiles + kTile * kLd;      // [state][token]
  const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
  float acc[4][4] = {};
  for (int s0 = 0; s0 < in.state; s0 += kTile) {
    const int width = min(kTile, in.state - s0);
    stage_columns(b_s, in.rows, in.stride, row0, n, in.b_off + group * in.state + s0, width);
    stage_columns(c_s, in.rows, in.stride, row0, n, in.c_off + group * in.state + s0, width);
    __syncthreads();
    tile_product(acc, by_query ? c_s : b_s, by_query ? b_s : c_s, width, ty, tx);
    __syncthreads();
  }
  float* dst = products + ((size_t)chunk * in.groups + group) * kChunk * kChunk;
#pragma unroll
  for (int a = 0; a < 4; ++a)
    *reinterpret_cast<float4*>(dst + (4 * ty + a) * kChunk + 4 * tx) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
}

// U of a (chunk, head), tile by tile of [state][vdim].  grid (chunks, groups + heads, state tiles * value tiles): the
// first `groups` rows of blocks work out G instead.
__global__ void __launch_bounds__(256)
ssd_chunk_sums_kernel(Inputs in, const float4* __restrict__ gates, float* __restrict__ products, float* __restrict__ sums,
                      const int* __restrict__ chunk_row, const int* __restrict__ chunk_count) {
  __shared__ __align__(16) float tiles[2 * kTile * kLd];
  __shared__ float w_s[kChunk];
  float *b_s = tiles, *x_s = tiles + kTile * kLd;      // [token][state], [token][value]
  pdl_wait();
  pdl_trigger();
  const int chunk = blockIdx.x, head = (int)blockIdx.y - in.groups;
  if (head < 0) {
    if (blockIdx.z == 0) chunk_products(in, products, chunk, blockIdx.y, chunk_row[chunk], chunk_count[chunk], false, tiles);
    return;
  }
  const int value_tiles = (in.vdim + kTile - 1) / kTile;
  const int s0 = blockIdx.z / value_tiles * kTile, v0 = blockIdx.z % value_tiles * kTile;
  const int row0 = chunk_row[chunk], n = chunk_count[chunk];
  const int group = head / (in.heads / in.groups);
  if (threadIdx.x < kChunk) {
    float w = 0.f;
    if (threadIdx.x < n) {
      const float4 g = gates[(size_t)(row0 + threadIdx.x) * in.heads + head];
      const float4 last = gates[(size_t)(row0 + n - 1) * in.heads + head];
      w = expf((last.y - g.y) + (last.z - g.z)) * g.x;
    }
    w_s[threadIdx.x] = w;
  }
  __syncthreads();
  stage_rows(b_s, in.rows, in.stride, row0, n, in.b_off + group * in.state + s0, min(kTile, in.state - s0), [&](int j) { return w_s[j]; });
  stage_rows(x_s, in.rows, in.stride, row0, n, in.x_off + head * in.vdim + v0, min(kTile, in.vdim - v0), [](int) { return 1.f; });
  __syncthreads();
  const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
  float acc[4][4] = {};
  tile_product(acc, b_s, x_s, n, ty, tx);
  float* dst = sums + ((size_t)chunk * in.heads + head) * in.state * in.vdim;
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    const int i = s0 + 4 * ty + a, c = v0 + 4 * tx;
    if (i >= in.state) continue;
    if (in.vdim % 4 == 0) {
      if (c < in.vdim) *reinterpret_cast<float4*>(dst + (size_t)i * in.vdim + c) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
    } else {
#pragma unroll
      for (int b = 0; b < 4; ++b)
        if (c + b < in.vdim) dst[(size_t)i * in.vdim + c + b] = acc[a][b];
    }
  }
}

// grid (requests, heads, blocks over state * vdim): a thread walks V neighbouring numbers of a head's state through the
// request's chunks.  decays: [chunks][heads], what a chunk leaves of the state before it.
template <int V>
__global__ void __launch_bounds__(128)
ssd_chunk_walk_kernel(float* __restrict__ sums, float* __restrict__ state, long long state_stride,
                      const float* __restrict__ decays, const int* __restrict__ request_chunk_start,
                      const int* __restrict__ slots, const int* __restrict__ request_active, int heads, int cells,
                      int max_slots, int* err) {
  pdl_wait();
  pdl_trigger();
  const int request = blockIdx.x, head = blockIdx.y;
  const int e = (blockIdx.z * blockDim.x + threadIdx.x) * V;
  if (e >= cells) return;
  const int slot = slots[request];
  if (slot < 0 || slot >= max_slots) {
    if (e == 0) atomicOr(err, kErrBadRequest);
    return;
  }
  float* cell = state + (size_t)slot * state_stride + (size_t)head * cells + e;
  float s[V];
  load_v<V>(s, cell);
  const size_t stride = (size_t)heads * cells;
  const int last = request_chunk_start[request + 1];
  constexpr int kBatch = 8;          // the sums of eight chunks are asked for together, before the first store
  for (int chunk = request_chunk_start[request]; chunk < last; chunk += kBatch) {
    float* u = sums + ((size_t)chunk * heads + head) * cells + e;
    float gained[kBatch][V], keep[kBatch];
#pragma unroll
    for (int b = 0; b < kBatch; ++b) {
      if (chunk + b >= last) break;
      load_v<V>(gained[b], u + b * stride);
      keep[b] = decays[(size_t)(chunk + b) * heads + head];
    }
#pragma unroll
    for (int b = 0; b < kBatch; ++b) {
      if (chunk + b >= last) break;
      store_v<V>(u + b * stride, s);
#pragma unroll
      for (int x = 0; x < V; ++x) s[x] = fmaf(keep[b], s[x], gained[b][x]);
    }
  }
  if (request_active[request]) store_v<V>(cell, s);
}

// grid (chunks, heads, value tiles)
__global__ void __launch_bounds__(256)
ssd_chunk_output_kernel(Inputs in, const float4* __restrict__ gates, const float* __restrict__ products,
                        const float* __restrict__ before_all, float* __restrict__ out, int out_stride,
                        const int* __restrict__ chunk_row, const int* __restrict__ chunk_count) {
  __shared__ __align__(16) float l_s[kTile * kLd], r_s[kTile * kLd];
  __shared__ float dt_s[kChunk], b_s[kChunk], rest_s[kChunk];
  pdl_wait();
  pdl_trigger();
  const int chunk = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * kTile;
  const int row0 = chunk_row[chunk], n = chunk_count[chunk];
  const int group = head / (in.heads / in.groups), width = min(kTile, in.vdim - v0);
  if (threadIdx.x < kChunk) {
    const float4 g = threadIdx.x < n ? gates[(size_t)(row0 + threadIdx.x) * in.heads + head] : make_float4(0.f, 0.f, 0.f, 0.f);
    dt_s[threadIdx.x] = g.x;
    b_s[threadIdx.x] = g.y;
    rest_s[threadIdx.x] = g.z;
  }
  const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
  const float* before = before_all + ((size_t)chunk * in.heads + head) * in.state * in.vdim;
  float acc[4][4] = {};
  for (int s0 = 0; s0 < in.state; s0 += kTile) {
    const int depth = min(kTile, in.state - s0);
    stage_columns(l_s, in.rows, in.stride, row0, n, in.c_off + group * in.state + s0, depth);
    stage_rows(r_s, before, in.vdim, s0, depth, v0, width, [](int) { return 1.f; });
    __syncthreads();
    tile_product(acc, l_s, r_s, depth, ty, tx);
    __syncthreads();
  }
  // what the state before the chunk gives decays to each token
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    const float carried = expf(b_s[4 * ty + a]);
#pragma unroll
    for (int b = 0; b < 4; ++b) acc[a][b] *= carried;
  }
  const float* g = products + ((size_t)chunk * in.groups + group) * kChunk * kChunk;
  for (int e = threadIdx.x; e < kChunk * kChunk; e += 256) {
    const int j = e / kChunk, i = e % kChunk;
    l_s[j * kLd + i] = (j <= i && i < n) ? g[e] * (expf((b_s[i] - b_s[j]) + (rest_s[i] - rest_s[j])) * dt_s[j]) : 0.f;
  }
  stage_rows(r_s, in.rows, in.stride, row0, n, in.x_off + head * in.vdim + v0, width, [](int) { return 1.f; });
  __syncthreads();
  tile_product(acc, l_s, r_s, min(n, (4 * ty + 7) & ~3), ty, tx);      // tokens up to this thread's last one
  const float skip = in.skip[head];
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    const int i = 4 * ty + a;
    if (i >= n) continue;
    float* dst = out + (size_t)(row0 + i) * out_stride + head * in.vdim + v0;
#pragma unroll
    for (int b = 0; b < 4; ++b)
      if (4 * tx + b < width) dst[4 * tx + b] = fmaf(skip, r_s[i * kLd + 4 * tx + b], acc[a][b]);
  }
}

// ---------------------------------------------------------------- chunks on the tensor cores
// Steps 3 and 5 with mma.sync (bfloat16 operands, float32 accumulators).  Every float32 operand enters as two bfloat16
// terms, its rounding and the rounding of what that left over, and of the four products of terms all but the smallest
// are taken: the operands are seen to within 2^-16 of their size.  Decays, rates, state and sums stay float32.
using bf16 = __nv_bfloat16;
constexpr int kPad = 8;          // elements behind a row: rows an odd number of 16-byte pieces apart

__device__ __forceinline__ unsigned smem_address(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_address(p)));
}
__device__ __forceinline__ void ldsm_trans(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_address(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// A tile as its two terms, COLS elements a row.
template <int COLS> struct Terms {
  static constexpr int ld = COLS + kPad, elements = kTile * ld;
  bf16 *hi, *lo;
  __device__ __forceinline__ explicit Terms(bf16* base) : hi(base), lo(base + elements) {}
  __device__ __forceinline__ void put(int row, int col, const float (&v)[4]) const {
    __align__(8) bf16 h[4], l[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      h[e] = __float2bfloat16_rn(v[e]);
      l[e] = __float2bfloat16_rn(v[e] - __bfloat162float(h[e]));
    }
    *reinterpret_cast<uint2*>(hi + row * ld + col) = *reinterpret_cast<const uint2*>(h);
    *reinterpret_cast<uint2*>(lo + row * ld + col) = *reinterpret_cast<const uint2*>(l);
  }
};

// 64 rows of COLS columns of float32 rows, times factor(row), as two terms; zero outside n rows and `width` columns.
template <int COLS, typename F>
__device__ __forceinline__ void stage_terms(const Terms<COLS>& dst, const float* src, int stride, int row0, int n, int col,
                                            int width, F factor) {
  const bool wide = ((reinterpret_cast<uintptr_t>(src + (size_t)row0 * stride + col) & 15) == 0) && stride % 4 == 0 && width % 4 == 0;
#pragma unroll 4
  for (int e = threadIdx.x; e < kTile * (COLS / 4); e += 256) {
    const int j = e / (COLS / 4), c = (e % (COLS / 4)) * 4;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (j < n && c < width) {
      const float* s = src + (size_t)(row0 + j) * stride + col + c;
      if (wide) {
        load_v<4>(v, s);
      } else {
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (c + x < width) v[x] = s[x];
      }
      const float f = factor(j);
#pragma unroll
      for (int x = 0; x < 4; ++x) v[x] *= f;
    }
    dst.put(j, c, v);
  }
}

// acc[16-column block][half][4] += A x B for one step of 16 along the sum; b points at row k of the right tile.
template <int NB, int COLS>
__device__ __forceinline__ void step_product(float (&acc)[NB][2][4], const uint32_t (&a_hi)[4], const uint32_t (&a_lo)[4],
                                             const Terms<COLS>& right, int k0, int n0, int lane) {
  const int mi = lane >> 3, r = lane & 7;
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) {
    const int at = (k0 + (mi & 1) * 8 + r) * Terms<COLS>::ld + n0 + nb * 16 + (mi >> 1) * 8;
    uint32_t hi[4], lo[4];
    ldsm_trans(hi, right.hi + at);
    ldsm_trans(lo, right.lo + at);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      mma(acc[nb][half], a_lo, hi[2 * half], hi[2 * half + 1]);
      mma(acc[nb][half], a_hi, lo[2 * half], lo[2 * half + 1]);
      mma(acc[nb][half], a_hi, hi[2 * half], hi[2 * half + 1]);
    }
  }
}

// U, MT state rows by 64 values a block; otherwise as ssd_chunk_sums_kernel.
template <int MT>
__global__ void __launch_bounds__(256)
ssd_chunk_sums_tensor_kernel(Inputs in, const float4* __restrict__ gates, float* __restrict__ products,
                             float* __restrict__ sums, const int* __restrict__ chunk_row, const int* __restrict__ chunk_count) {
  constexpr int kBytes = (2 * Terms<MT>::elements + 2 * Terms<kTile>::elements) * (int)sizeof(bf16);
  static_assert(kBytes >= 2 * kTile * kLd * (int)sizeof(float), "the products' tiles fit too");
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float w_s[kChunk];
  pdl_wait();
  pdl_trigger();
  const int chunk = blockIdx.x, head = (int)blockIdx.y - in.groups;
  const int row0 = chunk_row[chunk], n = chunk_count[chunk];
  if (head < 0) {
    if (blockIdx.z == 0) chunk_products(in, products, chunk, blockIdx.y, row0, n, true, reinterpret_cast<float*>(raw));
    return;
  }
  const Terms<MT> left(reinterpret_cast<bf16*>(raw));                                       // [token][state]
  const Terms<kTile> right(reinterpret_cast<bf16*>(raw) + 2 * Terms<MT>::elements);          // [token][value]
  const int value_tiles = (in.vdim + kTile - 1) / kTile;
  const int s0 = blockIdx.z / value_tiles * MT, v0 = blockIdx.z % value_tiles * kTile;
  const int group = head / (in.heads / in.groups);
  if (threadIdx.x < kChunk) {
    float w = 0.f;
    if (threadIdx.x < n) {
      const float4 g = gates[(size_t)(row0 + threadIdx.x) * in.heads + head];
      const float4 last = gates[(size_t)(row0 + n - 1) * in.heads + head];
      w = expf((last.y - g.y) + (last.z - g.z)) * g.x;
    }
    w_s[threadIdx.x] = w;
  }
  __syncthreads();
  stage_terms<MT>(left, in.rows, in.stride, row0, n, in.b_off + group * in.state + s0, min(MT, in.state - s0), [&](int j) { return w_s[j]; });
  stage_terms<kTile>(right, in.rows, in.stride, row0, n, in.x_off + head * in.vdim + v0, min(kTile, in.vdim - v0), [](int) { return 1.f; });
  __syncthreads();
  constexpr int kDown = MT / 16, kAcross = kWarps / kDown, kBlocks = kTile / kAcross / 16;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, r = lane & 7;
  const int m0 = (warp % kDown) * 16, n0 = (warp / kDown) * (kTile / kAcross);
  float acc[kBlocks][2][4] = {};
  const int steps = (n + 15) / 16;
  for (int k = 0; k < steps; ++k) {
    const int at = (k * 16 + (mi >> 1) * 8 + r) * Terms<MT>::ld + m0 + (mi & 1) * 8;      // stored [token][state]
    uint32_t a_hi[4], a_lo[4];
    ldsm_trans(a_hi, left.hi + at);
    ldsm_trans(a_lo, left.lo + at);
    step_product<kBlocks, kTile>(acc, a_hi, a_lo, right, k * 16, n0, lane);
  }
  float* dst = sums + ((size_t)chunk * in.heads + head) * in.state * in.vdim;
  const bool pairs = in.vdim % 2 == 0;
#pragma unroll
  for (int nb = 0; nb < kBlocks; ++nb)
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int i = s0 + m0 + (lane >> 2) + 8 * h, c = v0 + n0 + nb * 16 + half * 8 + 2 * (lane & 3);
        if (i >= in.state || c >= in.vdim) continue;
        float* d = dst + (size_t)i * in.vdim + c;
        if (pairs) {
          *reinterpret_cast<float2*>(d) = make_float2(acc[nb][half][2 * h], acc[nb][half][2 * h + 1]);
        } else {
          d[0] = acc[nb][half][2 * h];
          if (c + 1 < in.vdim) d[1] = acc[nb][half][2 * h + 1];
        }
      }
}

// Step 5; products as [i][j].  grid (chunks, heads, value tiles)
__global__ void __launch_bounds__(256)
ssd_chunk_output_tensor_kernel(Inputs in, const float4* __restrict__ gates, const float* __restrict__ products,
                               const float* __restrict__ before_all, float* __restrict__ out, int out_stride,
                               const int* __restrict__ chunk_row, const int* __restrict__ chunk_count) {
  __shared__ __align__(16) bf16 left_s[2 * Terms<kTile>::elements], right_s[2 * Terms<kTile>::elements];
  __shared__ float dt_s[kChunk], b_s[kChunk], rest_s[kChunk];
  const Terms<kTile> left(left_s), right(right_s);
  pdl_wait();
  pdl_trigger();
  const int chunk = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * kTile;
  const int row0 = chunk_row[chunk], n = chunk_count[chunk];
  const int group = head / (in.heads / in.groups), width = min(kTile, in.vdim - v0);
  if (threadIdx.x < kChunk) {
    const float4 g = threadIdx.x < n ? gates[(size_t)(row0 + threadIdx.x) * in.heads + head] : make_float4(0.f, 0.f, 0.f, 0.f);
    dt_s[threadIdx.x] = g.x;
    b_s[threadIdx.x] = g.y;
    rest_s[threadIdx.x] = g.z;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32;      // a warp: 16 tokens, 32 values
  const float* before = before_all + ((size_t)chunk * in.heads + head) * in.state * in.vdim;
  float acc[2][2][4] = {};
  auto multiply = [&](int steps) {
    for (int k = 0; k < steps; ++k) {
      const int at = (m0 + (lane & 15)) * Terms<kTile>::ld + k * 16 + (lane >> 4) * 8;
      uint32_t a_hi[4], a_lo[4];
      ldsm(a_hi, left.hi + at);
      ldsm(a_lo, left.lo + at);
      step_product<2, kTile>(acc, a_hi, a_lo, right, k * 16, n0, lane);
    }
  };
  for (int s0 = 0; s0 < in.state; s0 += kTile) {
    const int depth = min(kTile, in.state - s0);
    stage_terms<kTile>(left, in.rows, in.stride, row0, n, in.c_off + group * in.state + s0, depth, [](int) { return 1.f; });
    stage_terms<kTile>(right, before, in.vdim, s0, depth, v0, width, [](int) { return 1.f; });
    __syncthreads();
    multiply((depth + 15) / 16);
    __syncthreads();
  }
  const int i0 = m0 + (lane >> 2);
  const float carried[2] = {expf(b_s[i0]), expf(b_s[i0 + 8])};      // what the state before the chunk gives decays
#pragma unroll
  for (int nb = 0; nb < 2; ++nb)
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[nb][half][e] *= carried[e >> 1];
  const float* g = products + ((size_t)chunk * in.groups + group) * kChunk * kChunk;
#pragma unroll
  for (int e = threadIdx.x; e < kChunk * (kChunk / 4); e += 256) {
    const int i = e / (kChunk / 4), j = (e % (kChunk / 4)) * 4;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (j <= i && i < n) {
      load_v<4>(v, g + i * kChunk + j);
#pragma unroll
      for (int x = 0; x < 4; ++x) v[x] = j + x <= i ? v[x] * (expf((b_s[i] - b_s[j + x]) + (rest_s[i] - rest_s[j + x])) * dt_s[j + x]) : 0.f;
    }
    left.put(i, j, v);
  }
  stage_terms<kTile>(right, in.rows, in.stride, row0, n, in.x_off + head * in.vdim + v0, width, [](int) { return 1.f; });
  __syncthreads();
  multiply(min(m0 / 16 + 1, (n + 15) / 16));      // tokens up to this warp's last one
  const float skip = in.skip[head];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int i = i0 + 8 * h;
    if (i >= n) continue;
    const float* x = in.rows + (size_t)(row0 + i) * in.stride + in.x_off + head * in.vdim + v0;
    float* dst = out + (size_t)(row0 + i) * out_stride + head * in.vdim + v0;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int c = n0 + nb * 16 + half * 8 + 2 * (lane & 3) + y;
          if (c < width) dst[c] = fmaf(skip, x[c], acc[nb][half][2 * h + y]);
        }
  }
}

}  // namespace cie

using namespace cie;

extern "C" int cie_ssd_max_state() { return kMaxState; }
extern "C" int cie_ssd_chunk_tokens() { return kChunk; }

// rows: float32 rows with x (heads * vdim), B and C (groups * state each) at the given columns; proj: rows with the
// rates (heads) at r_off.  state: float32, slot after slot `state_stride` floats apart, heads [state][vdim] each.
extern "C" int cie_ssd_scan(const float* rows, int stride, int x_off, int b_off, int c_off, const float* proj,
                            int proj_stride, int r_off, const float* a_log, const float* dt_bias, const float* skip,
                            float* out, int out_stride, float* state, long long state_stride, const int* query_start,
                            const int* slots, const int* request_active, int requests, int heads, int groups, int n,
                            int vdim, int max_slots, int* err, void* stream) {
  if (requests <= 0) return 0;
  if (n < 1 || n > kMaxState) CIE_FAIL("ssd_scan: a state of %d rows is outside 1..%d", n, kMaxState);
  if (groups < 1 || heads < 1 || heads % groups || vdim < 1) CIE_FAIL("ssd_scan: %d heads of %d in %d groups", heads, vdim, groups);
  const Inputs in{rows, stride, x_off, b_off, c_off, proj, proj_stride, r_off, a_log, dt_bias, skip, heads, groups, n, vdim};
  const dim3 grid(requests, heads, (vdim + 31) / 32);
#define CIE_SSD_SCAN(R)                                                                                              \
  CIE_LAUNCH("ssd_scan", ssd_scan_kernel<R>, grid, dim3(kWarps * 32), 0, (cudaStream_t)stream, in, out, out_stride,  \
             state, state_stride, query_start, slots, request_active, max_slots, err)
  if (n <= 32) CIE_SSD_SCAN(4);
  else if (n <= 64) CIE_SSD_SCAN(8);
  else if (n <= 128) CIE_SSD_SCAN(16);
  else CIE_SSD_SCAN(32);
#undef CIE_SSD_SCAN
  return 0;
}

// Floats of scratch memory: gates, decays, products, sums.
extern "C" long long cie_ssd_chunk_floats(int tokens, int chunks, int heads, int groups, int n, int vdim) {
  const long long gates = (long long)4 * tokens * heads;
  const long long decays = ((long long)chunks * heads + 3) / 4 * 4;
  return gates + decays + (long long)chunks * groups * kChunk * kChunk + (long long)chunks * heads * n * vdim;
}

extern "C" int cie_ssd_chunked(const float* rows, int stride, int x_off, int b_off, int c_off, const float* proj,
                               int proj_stride, int r_off, const float* a_log, const float* dt_bias, const float* skip,
                               float* out, int out_stride, float* state, long long state_stride, float* scratch,
                               const int* chunk_row, const int* chunk_count, const int* request_chunk_start,
                               const int* slots, const int* request_active, int tokens, int chunks, int requests,
                               int heads, int groups, int n, int vdim, int max_slots, int tensor, int* err,
                               void* stream) {
  // tensor: 1 runs steps 3 and 5 with mma.sync on operands split into two bfloat16 terms, 0 on the CUDA cores
  if (chunks <= 0 || requests <= 0) return 0;
  if (n < 1 || vdim < 1) CIE_FAIL("ssd_chunked: a state of %d x %d", n, vdim);
  if (groups < 1 || heads < 1 || heads + groups > 65535 || heads % groups) CIE_FAIL("ssd_chunked: %d heads in %d groups", heads, groups);
  const Inputs in{rows, stride, x_off, b_off, c_off, proj, proj_stride, r_off, a_log, dt_bias, skip, heads, groups, n, vdim};
  cudaStream_t s = (cudaStream_t)stream;
  float4* gates = reinterpret_cast<float4*>(scratch);
  float* decays = scratch + (long long)4 * tokens * heads;
  float* products = decays + ((long long)chunks * heads + 3) / 4 * 4;
  float* sums = products + (size_t)chunks * groups * kChunk * kChunk;
  const int state_tiles = (n + kTile - 1) / kTile, value_tiles = (vdim + kTile - 1) / kTile;
  CIE_LAUNCH("ssd_gates", ssd_gates_kernel, dim3(chunks, (heads + 31) / 32), dim3(256), 0, s, in, gates, decays, chunk_row,
             chunk_count);
  if (tensor) {
#define CIE_SSD_SUMS(MT)                                                                                             \
  do {                                                                                                               \
    constexpr int smem = (2 * Terms<MT>::elements + 2 * Terms<kTile>::elements) * (int)sizeof(bf16);                  \
    static bool configured = false;                                                                                  \
    if (!configured) {                                                                                               \
      if (cudaFuncSetAttribute(ssd_chunk_sums_tensor_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != \
          cudaSuccess)                                                                                               \
        CIE_FAIL("ssd_chunked: cannot reserve %d bytes of shared memory", smem);                                     \
      configured = true;                                                                                             \
    }                                                                                                                \
    CIE_LAUNCH("ssd_chunk_sums", ssd_chunk_sums_tensor_kernel<MT>, dim3(chunks, groups + heads, (n + MT - 1) / MT * value_tiles), \
               dim3(256), smem, s, in, (const float4*)gates, products, sums, chunk_row, chunk_count);                 \
  } while (0)
    if (n > 64) CIE_SSD_SUMS(128);
    else CIE_SSD_SUMS(64);
#undef CIE_SSD_SUMS
  } else {
    CIE_LAUNCH("ssd_chunk_sums", ssd_chunk_sums_kernel, dim3(chunks, groups + heads, state_tiles * value_tiles), dim3(256), 0, s,
               in, (const float4*)gates, products, sums, chunk_row, chunk_count);
  }
  const int cells = n * vdim;
  const bool wide = cells % 4 == 0 && state_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
#define CIE_SSD_WALK(V)                                                                                              \
  CIE_LAUNCH("ssd_chunk_walk", ssd_chunk_walk_kernel<V>, dim3(requests, heads, (cells + 128 * V - 1) / (128 * V)),   \
             dim3(128), 0, s, sums, state, state_stride, (const float*)decays, request_chunk_start, slots,           \
             request_active, heads, cells, max_slots, err)
  if (wide) CIE_SSD_WALK(4);
  else CIE_SSD_WALK(1);
#undef CIE_SSD_WALK
  if (tensor)
    CIE_LAUNCH("ssd_chunk_output", ssd_chunk_output_tensor_kernel, dim3(chunks, heads, value_tiles), dim3(256), 0, s, in,
               (const float4*)gates, (const float*)products, (const float*)sums, out, out_stride, chunk_row, chunk_count);
  else
    CIE_LAUNCH("ssd_chunk_output", ssd_chunk_output_kernel, dim3(chunks, heads, value_tiles), dim3(256), 0, s, in,
               (const float4*)gates, (const float*)products, (const float*)sums, out, out_stride, chunk_row, chunk_count);
  return 0;
}

// Attention of prompt portions over a cached latent, with keys and values EXPANDED, on the 5th-generation tensor cores
// (bfloat16 pages; latent.cu has the arithmetic, and serves single tokens without expanding anything).
//
// For a portion of many tokens it is cheaper to work out every head's keys and values of the portion's context once
// (W_uk c, W_uv c: one library product over the gathered latents) and to attend over heads of dim + rot and vdim
// elements than to attend over latents of rank + rot elements for every (token, head).
//
//   latent_gather     the cached rows a step's portions can see, request after request, out of the pages: latents
//                     [keys][rank] and rotated key parts [keys][rot]
//   latent_queries    the queries, float32, rounded to bfloat16 once, their rotated part after the rotation; every part of
//                     a head padded with zeros to whole steps of 16
//   latent_prompt     softmax attention of 128 tokens of one request and one head a CTA over its expanded rows
//
// In a CTA of latent_prompt keys go by in tiles of 128:
//
//   TMA thread        key tiles (the head's columns of the expanded rows, and the shared rotated key parts) and value
//                     tiles into two stages each, 64-column pieces in the 128-byte swizzle
//   MMA thread        S = Q K^T (128 x 128, float32, tensor memory, two buffers) and O += P V
//   2 x 4 softmax     one group takes the even tiles, the other the odd ones, each with a running maximum, a sum and an
//   warps             accumulator O of its own; a thread owns a row: it reads S, and writes P over it in tensor memory
//                     as TWO bfloat16 terms (the weight rounded, and what the rounding left), both multiplied with V
//                     from there.  Maxima, sums and denominators are float32.  At the end the groups' halves join.
//
// Options: a window, a sink term in the denominator, a gate on the result.  Every wait on an mbarrier is bounded.  A
// row's result depends on its own request's rows alone.
#include "blackwell.cuh"
#include "common.cuh"

#include <cfloat>

CIE_DEFINE_LAST_ERROR()

namespace cie {

using namespace bw;
using bf16 = __nv_bfloat16;

constexpr int BM = 128, BN = 128;          // query rows of a CTA, keys of a tile
constexpr int PIECE = 64;                  // columns of a swizzled piece
constexpr int PIECE_BYTES = 128 * 128;     // 128 rows of 64 columns
constexpr int STAGES = 2;
constexpr int MMA_WARP = 8, TMA_WARP = 9;
constexpr int THREADS = 320;
constexpr int TMEM_COLS = 512;             // S0 | S1 | O0 | O1, 128 columns each
constexpr uint32_t COL_S = 0, COL_O = 256;
constexpr float kGrow = 8.f;               // rescale O when a maximum moved by more than this (log2 units)
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float fast_exp2(float x) {      // results below 2^-126 become 0; -inf gives 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ uint32_t pack(float a, float b) {
  const __nv_bfloat162 pair = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&pair);
}

// Behind tcgen05.wait::ld: what is done with these registers stays behind it too.
__device__ __forceinline__ void pin(uint32_t (&r)[32]) {
#pragma unroll
  for (int i = 0; i < 32; ++i) asm volatile("" : "+r"(r[i]));
}

// ---------------------------------------------------------------- gather
// portions: (request, first row, first key) of every portion, rows ascending, then (.., rows in all, ..); block_portion[b]:
// the portion that row 128 b belongs to.  A warp a row; rows beyond the last are zeros.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const bf16* __restrict__ c_pool, const bf16* __restrict__ r_pool, const int* __restrict__ portions,
                     int count, const int* __restrict__ block_portion, const int* __restrict__ table, int table_width,
                     int num_pages, int page_size, int rank, int rot, bf16* __restrict__ c_rows, bf16* __restrict__ r_rows,
                     int rows, int* err) {
  const int row = blockIdx.x * (blockDim.x / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  pdl_wait();
  pdl_trigger();
  const uint4* c_src = nullptr;
  const uint4* r_src = nullptr;
  if (row < portions[3 * count + 1]) {
    int p = block_portion[row / 128];
    while (row >= portions[3 * (p + 1) + 1]) ++p;            // ends at the last portion: row lies below the total
    const int key = portions[3 * p + 2] + row - portions[3 * p + 1];
    const int page = key / page_size < table_width ? table[(size_t)portions[3 * p] * table_width + key / page_size] : -1;
    if (page < 0 || page >= num_pages) {
      if (lane == 0) atomicOr(err, kErrBadPage);
    } else {
      const size_t slot = (size_t)page * page_size + key % page_size;
      c_src = reinterpret_cast<const uint4*>(c_pool + slot * rank);
      r_src = reinterpret_cast<const uint4*>(r_pool + slot * rot);
    }
  }
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4* c_dst = reinterpret_cast<uint4*>(c_rows + (size_t)row * rank);
  uint4* r_dst = reinterpret_cast<uint4*>(r_rows + (size_t)row * rot);
  for (int i = lane; i < rank / 8; i += 32) c_dst[i] = c_src ? c_src[i] : zero;
  for (int i = lane; i < rot / 8; i += 32) r_dst[i] = r_src ? r_src[i] : zero;
}

// ---------------------------------------------------------------- queries
__host__ __device__ __forceinline__ int padded16(int columns) { return (columns + 15) / 16 * 16; }

// A block per token: q [heads * (dim + rot)] float32 -> out [heads * (padded dim + padded rot)], 8 elements a thread at a time.
constexpr int kMaxPairs = 128;
__global__ void __launch_bounds__(256)
latent_queries_kernel(const float* __restrict__ q, int q_stride, bf16* __restrict__ out, const int* __restrict__ positions,
                      const float* __restrict__ inv_freq, float magnitude, int interleaved, int rot_dims, int heads, int dim,
                      int rot) {
  __shared__ float sin_s[kMaxPairs], cos_s[kMaxPairs];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x, half = rot_dims / 2, plain = padded16(dim), width = plain + padded16(rot);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf((float)positions[t] * inv_freq[i], &s, &c);
    sin_s[i] = s * magnitude;
    cos_s[i] = c * magnitude;
  }
  __syncthreads();
  const float* row = q + (size_t)t * q_stride;
  uint4* dst = reinterpret_cast<uint4*>(out + (size_t)t * heads * width);
  const int per_head = width / 8;
  for (int piece = threadIdx.x; piece < heads * per_head; piece += blockDim.x) {
    const int h = piece / per_head, column = (piece - h * per_head) * 8;
    const float* src = row + (size_t)h * (dim + rot) + (column < plain ? column : dim + column - plain);
    float v[8] = {};
    const int first = column - plain;                       // in the rotated part
    if (first < 0 ? column < dim : first < rot) {           // dim and rot are multiples of 8
      const float4 lo = reinterpret_cast<const float4*>(src)[0], hi = reinterpret_cast<const float4*>(src)[1];
      v[0] = lo.x; v[1] = lo.y; v[2] = lo.z; v[3] = lo.w;
      v[4] = hi.x; v[5] = hi.y; v[6] = hi.z; v[7] = hi.w;
      if (first >= 0) {
        if (interleaved) {
#pragma unroll
          for (int e = 0; e < 8; e += 2) {
            if (first + e >= rot_dims) continue;
            const float u = v[e], w = v[e + 1], s = sin_s[(first + e) / 2], c = cos_s[(first + e) / 2];
            v[e] = u * c - w * s;
            v[e + 1] = w * c + u * s;
          }
        } else {
          const float* part = row + (size_t)h * (dim + rot) + dim;
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const int d = first + e;
            if (d >= rot_dims) continue;
            const int i = d < half ? d : d - half;
            const float other = part[d < half ? d + half : d - half];
            v[e] = d < half ? v[e] * cos_s[i] - other * sin_s[i] : v[e] * cos_s[i] + other * sin_s[i];
          }
        }
      }
    }
    dst[piece] = make_uint4(pack(v[0], v[1]), pack(v[2], v[3]), pack(v[4], v[5]), pack(v[6], v[7]));
  }
}

// ---------------------------------------------------------------- attention
struct PromptArgs {
  bf16* out;                 // token t, head h at out[t * out_stride + h * vdim]
  int out_stride;
  const float* gate;         // like out (gate_stride), or nullptr
  int gate_stride;
  const float* sink;         // [heads] or nullptr
  const int* tiles;          // (request, first token of the tile in the portion, first row, first key) per query tile
  const int* context_lens;
  const int* query_lens;
  const int* query_start;
  int token0;                // the token that row 0 of the queries belongs to
  int head0;                 // first head of this launch (its columns of the expanded rows start at 0)
  int dim, rot, vdim;
  int window;
  float scale_log2;
  int* err;
};

__host__ __device__ __forceinline__ int pieces_of(int columns) { return (columns + PIECE - 1) / PIECE; }

__global__ void __launch_bounds__(THREADS, 1)
latent_prompt_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap kv_map,
                     const __grid_constant__ CUtensorMap r_map, const PromptArgs a) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int k_plain = pieces_of(a.dim), k_pieces = k_plain + pieces_of(a.rot), v_pieces = pieces_of(a.vdim);
  const int k_bytes = k_pieces * PIECE_BYTES, v_bytes = v_pieces * PIECE_BYTES;
  unsigned char* q_s = smem;
  unsigned char* k_s = q_s + k_bytes;                  // [STAGES][k_bytes]
  unsigned char* v_s = k_s + STAGES * k_bytes;         // [STAGES][v_bytes]
  __shared__ __align__(8) uint64_t k_full[STAGES], k_empty[STAGES], v_full[STAGES], v_empty[STAGES];
  __shared__ __align__(8) uint64_t q_full, s_full[2], p_full[2], pv_done[2];
  __shared__ uint32_t tmem_slot;
  __shared__ float m_s[2][BM], l_s[2][BM];

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int head = a.head0 + blockIdx.x;
  if (tid == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1);
    }
    mbar_init(&q_full, 1);
    for (int g = 0; g < 2; ++g) { mbar_init(&s_full[g], 1); mbar_init(&p_full[g], BM); mbar_init(&pv_done[g], 1); }
    mbar_init_fence();
  }
  pdl_wait();
  pdl_trigger();
  const int* tile = a.tiles + 4 * blockIdx.y;          // the list puts the tiles with the most keys first, all heads of each
  const int request = tile[0], q0 = tile[1], row0 = tile[2], key0 = tile[3];
  const int q_len = a.query_lens[request], first_token = a.query_start[request] + q0;
  const int ntok = min(BM, q_len - q0);
  // keys are counted from the request's first expanded row: row i is key key0 + i
  const int pos_lo = a.context_lens[request] + q0 - key0;         // the first query's own key
  const int valid_hi = pos_lo + ntok;                             // keys [.., valid_hi) are visible to some row
  const int lowest = a.window > 0 ? max(0, pos_lo + 1 - a.window) : 0;
  const int tile0 = lowest / BN, tiles = (valid_hi + BN - 1) / BN - tile0;

  if (warp == MMA_WARP) tmem_alloc<TMEM_COLS>(&tmem_slot);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;

  bool alive = true;
  if (warp == TMA_WARP) {
    if (lane == 0) {
      const int column = blockIdx.x * (a.dim + a.vdim);
      // the queries: plain part and rotated part begin at pieces of their own; what a piece holds beyond a part's padded
      // columns takes part in no product
      const int q_column = head * (padded16(a.dim) + padded16(a.rot)), q_row = first_token - a.token0;
      mbar_expect_tx(&q_full, (uint32_t)k_bytes);
      for (int p = 0; p < k_pieces; ++p)
        tma_load_2d(q_s + p * PIECE_BYTES, &q_map, &q_full,
                    q_column + (p < k_plain ? p * PIECE : padded16(a.dim) + (p - k_plain) * PIECE), q_row);
      for (int j = 0; j < tiles; ++j) {
        const int s = j % STAGES, row = row0 + (tile0 + j) * BN;
        const uint32_t before = ((j / STAGES) - 1) & 1;
        if (j >= STAGES && !mbar_wait(&k_empty[s], before, a.err)) { alive = false; break; }
        mbar_expect_tx(&k_full[s], (uint32_t)k_bytes);       // a whole box counts, also where it reaches past the matrix
        for (int p = 0; p < k_plain; ++p)
          tma_load_2d(k_s + s * k_bytes + p * PIECE_BYTES, &kv_map, &k_full[s], column + p * PIECE, row);
        for (int p = k_plain; p < k_pieces; ++p)
          tma_load_2d(k_s + s * k_bytes + p * PIECE_BYTES, &r_map, &k_full[s], (p - k_plain) * PIECE, row);
        if (j >= STAGES && !mbar_wait(&v_empty[s], before, a.err)) { alive = false; break; }
        mbar_expect_tx(&v_full[s], (uint32_t)v_bytes);
        for (int p = 0; p < v_pieces; ++p)
          tma_load_2d(v_s + s * v_bytes + p * PIECE_BYTES, &kv_map, &v_full[s], column + a.dim + p * PIECE, row);
      }
    }
    __syncwarp();
  } else if (warp == MMA_WARP) {
    if (lane == 0) {
      constexpr uint32_t idesc_qk = idesc_bf16(BM, BN);
      const uint32_t idesc_pv = idesc_bf16(BM, (a.vdim + 15) / 16 * 16, true);
      const uint64_t q_desc = smem_desc_sw128(smem_u32(q_s)), k_desc0 = smem_desc_sw128(smem_u32(k_s));
      // values: the operand whose N dimension is contiguous, 64-column pieces PIECE_BYTES apart
      const uint64_t v_desc0 = smem_desc_sw128(smem_u32(v_s), PIECE_BYTES);
      const int plain_steps = (a.dim + 15) / 16, rot_steps = (a.rot + 15) / 16;
      auto values = [&](int j) -> bool {
        const int g = j & 1, s = j % STAGES;
        if (!mbar_wait(&p_full[g], (j >> 1) & 1, a.err) || !mbar_wait(&v_full[s], (j / STAGES) & 1, a.err)) return false;
        tc_fence_after();
        const uint64_t v_desc = v_desc0 + (uint64_t)((s * v_bytes) >> 4);
#pragma unroll
        for (int kk = 0; kk < BN / 16; ++kk) {
          // P lies over S: 32 columns hold 32 keys, 16 columns of first terms and then 16 of second ones
          const uint32_t p = tmem + COL_S + g * BN + (kk >> 1) * 32 + (kk & 1) * 8;
          const uint64_t v = v_desc + (uint64_t)((kk * 2048) >> 4);
          umma_bf16_ta(tmem + COL_O + g * 128, p, v, idesc_pv, (j > 1 || kk > 0) ? 1u : 0u);
          umma_bf16_ta(tmem + COL_O + g * 128, p + 16, v, idesc_pv, 1u);
        }
        tc_commit(&v_empty[s]);
        tc_commit(&pv_done[g]);
        return true;
      };
      alive = mbar_wait(&q_full, 0, a.err);
      for (int j = 0; j < tiles && alive; ++j) {
        const int g = j & 1, s = j % STAGES;
        // the weights of tile j - 2, which lie in this buffer, have been used
        if (j > 1 && !mbar_wait(&pv_done[g], ((j >> 1) - 1) & 1, a.err)) { alive = false; break; }
        if (!mbar_wait(&k_full[s], (j / STAGES) & 1, a.err)) { alive = false; break; }
        tc_fence_after();
        const uint64_t k_desc = k_desc0 + (uint64_t)((s * k_bytes) >> 4);
        for (int kk = 0; kk < plain_steps + rot_steps; ++kk) {
          const int at = kk < plain_steps ? kk : k_plain * 4 + kk - plain_steps;       // in steps of 16 columns
          const uint32_t offset = (uint32_t)((at >> 2) * PIECE_BYTES + (at & 3) * 32) >> 4;
          umma_bf16(tmem + COL_S + g * BN, q_desc + offset, k_desc + offset, idesc_qk, kk > 0 ? 1u : 0u);
        }
        tc_commit(&s_full[g]);
        tc_commit(&k_empty[s]);
        if (j > 0) alive = values(j - 1);
      }
      if (alive) alive = values(tiles - 1);
    }
    __syncwarp();
  } else {
    // ---- softmax: group g takes tiles g, g + 2, ..; thread r of a group owns row r = tensor-memory lane r
    const int g = warp >> 2, r = tid & 127;
    const int pos = r < ntok ? pos_lo + r : -1;
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t s_addr = tmem + lane_base + COL_S + g * BN, o_addr = tmem + lane_base + COL_O;
    const int o_chunks = (a.vdim + 31) / 32;
    float m_used = -INFINITY, l = 0.f;
    for (int j = g; j < tiles; j += 2) {
      if (!mbar_wait(&s_full[g], (j >> 1) & 1, a.err)) { alive = false; break; }
      tc_fence_after();
      const int k0 = (tile0 + j) * BN;
      const int hi = pos - k0;                                           // columns lo .. hi of this tile are visible
      const int lo = a.window > 0 ? hi - a.window + 1 : 0;
      const bool masked = k0 + BN - 1 > pos_lo || (a.window > 0 && k0 < valid_hi - a.window);      // the same for the CTA
      // the row of S comes twice: for its maximum, and, 32 columns at a time, for the weights
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      uint32_t raw[2][32];
      {
        uint32_t all[BN / 32][32];
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) tmem_ld32(s_addr + c * 32, all[c]);
        tc_wait_ld();
        if (masked) {
#pragma unroll
          for (int i = 0; i < BN; ++i) {
            if (i > hi || i < lo) all[i >> 5][i & 31] = 0xff800000u;      // -inf: out of the maximum
            mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(all[i >> 5][i & 31]));
          }
        } else {
#pragma unroll
          for (int i = 0; i < BN; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(all[i >> 5][i & 31]));
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) raw[0][i] = all[0][i];
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * a.scale_log2;
      const bool grow = mx > m_used + kGrow;            // false while the row has seen no key
      if (__any_sync(0xffffffffu, grow)) {
        float alpha = 1.f;
        if (grow) {
          alpha = exp2f(m_used - mx);                   // 0 at the row's first keys
          m_used = mx;
          l *= alpha;
        }
        if (j > 1) {
          // S of this tile was asked for after O += P V of the group's tile before it had ended: O stands still
          for (int c = 0; c < o_chunks; ++c) {
            uint32_t raw[32];
            tmem_ld32(o_addr + g * 128 + c * 32, raw);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) raw[i] = __float_as_uint(__uint_as_float(raw[i]) * alpha);
            tmem_st32(o_addr + g * 128 + c * 32, raw);
          }
        }
      }
      const float m_eff = m_used == -INFINITY ? 0.f : m_used;
      float l4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < BN / 32; ++c) {
        uint32_t terms[32];
        uint32_t (&here)[32] = raw[c & 1];
        if (c > 0) {
          tc_wait_ld();
          pin(here);
          if (masked) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (c * 32 + i > hi || c * 32 + i < lo) here[i] = 0xff800000u;      // -inf: a weight of 0
          }
        }
        if (c + 1 < BN / 32) tmem_ld32(s_addr + (c + 1) * 32, raw[(c + 1) & 1]);     // on its way while this one is used
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float p0 = fast_exp2(fmaf(__uint_as_float(here[i]), a.scale_log2, -m_eff));
          const float p1 = fast_exp2(fmaf(__uint_as_float(here[i + 1]), a.scale_log2, -m_eff));
          l4[(i >> 1) & 3] += p0 + p1;
          const __nv_bfloat162 first = __floats2bfloat162_rn(p0, p1);
          const float2 back = __bfloat1622float2(first);
          const __nv_bfloat162 second = __floats2bfloat162_rn(p0 - back.x, p1 - back.y);
          terms[i >> 1] = *reinterpret_cast<const uint32_t*>(&first);
          terms[16 + (i >> 1)] = *reinterpret_cast<const uint32_t*>(&second);
        }
        tmem_st32(s_addr + c * 32, terms);
      }
      l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
      tc_wait_st();
      tc_fence_before();
      mbar_arrive(&p_full[g]);
    }
    // ---- the groups' halves: each group finishes half of the columns of every row
    const int mine = (tiles - g + 1) / 2;               // tiles of this group
    if (alive && mine > 0 && !mbar_wait(&pv_done[g], (mine - 1) & 1, a.err)) alive = false;
    tc_fence_after();
    m_s[g][r] = alive ? m_used : -INFINITY;
    l_s[g][r] = l;
    tc_fence_before();
    asm volatile("bar.sync 1, 256;" ::: "memory");
    tc_fence_after();
    const float m0 = m_s[0][r], m1 = m_s[1][r];
    float top = fmaxf(m0, m1), sink = 0.f;
    if (a.sink) {
      sink = a.sink[head] * kLog2e;
      top = fmaxf(top, sink);
    }
    const float w0 = m0 == -INFINITY ? 0.f : exp2f(m0 - top), w1 = m1 == -INFINITY ? 0.f : exp2f(m1 - top);
    float total = l_s[0][r] * w0 + l_s[1][r] * w1;
    if (a.sink) total += exp2f(sink - top);
    const float inv = total > 0.f ? 1.f / total : 0.f;
    const bool both = tiles > 1;
    bf16* dst = a.out + (size_t)(first_token + r) * a.out_stride + (size_t)head * a.vdim;
    const float* gate = a.gate ? a.gate + (size_t)(first_token + r) * a.gate_stride + (size_t)head * a.vdim : nullptr;
    for (int c = g; c < o_chunks; c += 2) {
      uint32_t x0[32], x1[32];
      tmem_ld32(o_addr + c * 32, x0);
      if (both) tmem_ld32(o_addr + 128 + c * 32, x1);
      tc_wait_ld();
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        const int column = c * 32 + p * 8;
        if (r >= ntok || column >= a.vdim) continue;    // vdim is a multiple of 8
        float o[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          o[e] = __uint_as_float(x0[p * 8 + e]) * w0;
          if (both) o[e] = fmaf(__uint_as_float(x1[p * 8 + e]), w1, o[e]);
          o[e] *= inv;
          if (gate) o[e] *= 1.f / (1.f + expf(-gate[column + e]));
        }
        *reinterpret_cast<uint4*>(dst + column) = make_uint4(pack(o[0], o[1]), pack(o[2], o[3]), pack(o[4], o[5]), pack(o[6], o[7]));
      }
      __syncwarp();
    }
  }
  if (!alive)      // a wait ran out: give copies and products that may still be in flight time to end before leaving
    for (int i = 0; i < 1000; ++i) __nanosleep(1000);
  tc_fence_before();
  __syncthreads();
  if (warp == MMA_WARP) tmem_free<TMEM_COLS>(tmem);
}

}  // namespace cie

using namespace cie;

static size_t prompt_smem(int dim, int rot, int vdim) {
  const int k = pieces_of(dim) + pieces_of(rot), v = pieces_of(vdim);
  return (size_t)((1 + STAGES) * k + STAGES * v) * PIECE_BYTES + 1024;
}

// 1 if the kernels take these sizes (bfloat16).
extern "C" int cie_latent_prompt_supports(int dim, int rot, int vdim, int rank) {
  return dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && rank % 8 == 0 && dim >= 8 && rot >= 8 && vdim >= 8 && rank >= 8 &&
         vdim <= 128 && prompt_smem(dim, rot, vdim) <= 220 * 1024 ? 1 : 0;
}

extern "C" int cie_latent_gather(const void* c_pool, const void* r_pool, const int* portions, int count,
                                 const int* block_portion, const int* table, int table_width, int num_pages, int page_size,
                                 int rank, int rot, void* c_rows, void* r_rows, int rows, int* err, void* stream) {
  if (rows <= 0 || count <= 0) return 0;
  if (rows % 128 || rank % 8 || rot % 8) CIE_FAIL("latent_gather: %d rows of %d and %d elements", rows, rank, rot);
  CIE_LAUNCH("latent_gather", latent_gather_kernel, dim3(rows / 8), dim3(256), 0, (cudaStream_t)stream, (const bf16*)c_pool,
             (const bf16*)r_pool, portions, count, block_portion, table, table_width, num_pages, page_size, rank, rot,
             (bf16*)c_rows, (bf16*)r_rows, rows, err);
  return 0;
}

// q: float32, token t, head h at q[t * q_stride + h * (dim + rot)]: [dim plain | rot not yet rotated]; out: [tokens][heads *
// (dim padded to 16 + rot padded to 16)].
extern "C" int cie_latent_queries(const float* q, int q_stride, void* out, const int* positions, const float* inv_freq,
                                  float magnitude, int interleaved, int rot_dims, int tokens, int heads, int dim, int rot,
                                  void* stream) {
  if (tokens <= 0) return 0;
  if (dim % 8 || rot % 8 || q_stride % 4 || ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out)) & 15))
    CIE_FAIL("latent_queries: rows of heads of %d + %d elements must be 16-byte aligned", dim, rot);
  if (rot_dims % 2 || rot_dims > rot || rot_dims / 2 > kMaxPairs) CIE_FAIL("latent_queries: %d rotated dims of %d", rot_dims, rot);
  CIE_LAUNCH("latent_queries", latent_queries_kernel, dim3(tokens), dim3(256), 0, (cudaStream_t)stream, q, q_stride, (bf16*)out,
             positions, inv_freq, magnitude, interleaved, rot_dims, heads, dim, rot);
  return 0;
}

// queries: what latent_queries made of the tokens from token0 on (`tokens` rows, all_heads heads); kv_rows: [rows][heads *
// (dim + vdim)], per head its keys and then its values, for heads head0 .. head0 + heads - 1;
// r_rows: [rows][rot]; rows a multiple of 128.  tiles: [count][4] (see PromptArgs).
extern "C" int cie_latent_prompt(const void* queries, int tokens, int all_heads, int token0, void* out, int out_stride, const float* gate, int gate_stride,
                                 const float* sink, const void* kv_rows, const void* r_rows, int rows, const int* tiles,
                                 int count, const int* context_lens, const int* query_lens, const int* query_start,
                                 int head0, int heads, int dim, int rot, int vdim, int window, float scale, int* err, void* stream) {
  if (count <= 0 || heads <= 0) return 0;
  if (!cie_latent_prompt_supports(dim, rot, vdim, 8)) CIE_FAIL("latent_prompt: sizes %d + %d, %d", dim, rot, vdim);
  if (head0 < 0 || head0 + heads > all_heads) CIE_FAIL("latent_prompt: heads %d.. of %d", head0, all_heads);
  if (rows % 128 || out_stride % 8 || count > 65535) CIE_FAIL("latent_prompt: %d rows, stride %d, %d tiles", rows, out_stride, count);
  if ((reinterpret_cast<uintptr_t>(kv_rows) | reinterpret_cast<uintptr_t>(r_rows) | reinterpret_cast<uintptr_t>(out) |
       reinterpret_cast<uintptr_t>(queries)) & 15)
    CIE_FAIL("latent_prompt: operands must be 16-byte aligned");
  CUtensorMap q_map, kv_map, r_map;
  if (!tensor_map_bf16(queries, tokens, (long long)all_heads * (padded16(dim) + padded16(rot)), BM, &q_map) ||
      !tensor_map_bf16(kv_rows, rows, (long long)heads * (dim + vdim), BN, &kv_map) ||
      !tensor_map_bf16(r_rows, rows, rot, BN, &r_map))
    CIE_FAIL("latent_prompt: cuTensorMapEncodeTiled failed");
  const size_t smem = prompt_smem(dim, rot, vdim);
  static bool raised = false;
  if (!raised) {
    if (cudaFuncSetAttribute(latent_prompt_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess)
      CIE_FAIL("latent_prompt: cannot raise the shared memory limit");
    raised = true;
  }
  const PromptArgs a{(bf16*)out, out_stride, gate, gate_stride, sink, tiles, context_lens, query_lens, query_start,
                     token0, head0, dim, rot, vdim, window, scale * kLog2e, err};
  CIE_LAUNCH("latent_prompt", latent_prompt_kernel, dim3(heads, count), dim3(THREADS), smem, (cudaStream_t)stream, q_map,
             kv_map, r_map, a);
  return 0;
}

// RMS norms whose row is split into equal consecutive parts ("groups"), each divided by its OWN root mean square,
// and what sits right beside them in a layer:
//
//  * group_norm        the pending update joins the float32 stream, then the norm: out = gain * (x / rms of its part).
//                      The update is a sum of float32 terms (plain, or weighted by a number per row and term: a
//                      token's expert outputs), or such a sum that is itself RMS-normalised over the
//                      whole row and multiplied by a gain vector before it is added (`update_gain`).
//  * stream_rows       the same add, and the stream's own rows rounded to the activation type (no norm)
//  * group_norm_conv   the same norm followed by a causal convolution over time on every channel whose result is
//                      added to its input: with h the normalised rows,
//                          out_t = h_t + sum_j w[c][j] h_(t - taps + 1 + j)
//                      (zeros before a request's first token; h of the last taps - 1 tokens is the request's state).
//                      Single tokens: one kernel.  Prompt portions: add + statistics, convolution, history.
//  * gated_group_norm  u = y * silu(z), then every part of u by its own root mean square, times a gain
//  * side_gate         gelu_tanh(z) * a slice of a table row chosen by the token
//
// All sums, statistics and the stream are float32; a result is rounded once.  A row's result depends on that row
// (and the rows its convolution reads) alone.
#include "common.cuh"

CIE_DEFINE_LAST_ERROR()

namespace cie {

constexpr int kMaxTaps = 16;     // longest convolution
constexpr int kMaxTerms = 32;    // float32 terms of a pending update
constexpr int kMaxWarps = 32;

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// 0.5 z (1 + tanh(u)) with u = sqrt(2 / pi) (z + 0.044715 z^3), as z sigmoid(2 u): the same function without the
// cancellation of 1 + tanh for negative z, which a norm of the results would blow up.
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return z / (1.f + expf(-2.f * 0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
}

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
template <int V> __device__ __forceinline__ void store_v(__nv_bfloat16* dst, const float (&v)[V]) {
  if constexpr (V == 4) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  } else {
    dst[0] = __float2bfloat16_rn(v[0]);
  }
}

// How the threads of a block share a row: every part belongs to `wpg` warps (all parts at once), or, with more
// parts than warps, a warp takes one part after the other (wpg == 1).  A thread meets the same elements in
// every pass.
struct Share {
  int part, groups, wpg;
  template <int V, typename F> __device__ __forceinline__ void each(F f) const {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, step = (blockDim.x >> 5) / wpg;
    for (int g = warp / wpg; g < groups; g += step)
      for (int i = ((warp % wpg) * 32 + lane) * V; i < part; i += wpg * 32 * V) f(g, g * part + i);
  }
};

// inv_s[g] = 1 / sqrt(mean of the part's squares + eps) for every part of the row u_s; ends with a barrier.
template <int V>
__device__ __forceinline__ void part_inverses(const Share& share, const float* u_s, float* inv_s, float* warp_s, float eps) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, step = (blockDim.x >> 5) / share.wpg;
  for (int g = warp / share.wpg; g < share.groups; g += step) {
    float sq = 0.f;
    for (int i = ((warp % share.wpg) * 32 + lane) * V; i < share.part; i += share.wpg * 32 * V)
#pragma unroll
      for (int x = 0; x < V; ++x) sq = fmaf(u_s[g * share.part + i + x], u_s[g * share.part + i + x], sq);
    sq = warp_sum(sq);
    if (lane == 0) {
      if (share.wpg == 1) inv_s[g] = rsqrtf(sq / (float)share.part + eps);
      else warp_s[warp] = sq;
    }
  }
  __syncthreads();
  if (share.wpg > 1) {
    if (threadIdx.x < share.groups) {
      float total = 0.f;
      for (int k = 0; k < share.wpg; ++k) total += warp_s[threadIdx.x * share.wpg + k];
      inv_s[threadIdx.x] = rsqrtf(total / (float)share.part + eps);
    }
    __syncthreads();
  }
}

struct Update {
  const float* data;      // float32 terms: term s of row r at r * row_stride + s * stride; nullptr: nothing pending
  int terms;
  size_t stride, row_stride;
  const float* weights;   // not null: term s of row r is multiplied by weights[r * terms + s]
  const float* gain;      // not null: the sum is RMS-normalised over the whole row and multiplied by this first
  float eps;
};

// The row of the stream with its update applied, in u_s (and in the stream, unless write_back is false).
template <int V>
__device__ __forceinline__ void stream_row(const Share& share, float* residual, const Update& update, int row,
                                           bool write_back, float* u_s, float* scratch) {
  const int hidden = share.part * share.groups;
  float* res = residual + (size_t)row * hidden;
  if (update.data == nullptr) {
    share.each<V>([&](int, int i) {
      float x[V];
      load_v<V>(x, res + i);
      store_v<V>(u_s + i, x);
    });
    return;
  }
  const float* up = update.data + (size_t)row * update.row_stride;
  const float* weights = update.weights ? update.weights + (size_t)row * update.terms : nullptr;
  auto pending = [&](int i, float (&y)[V]) {
    load_v<V>(y, up + i);
    if (weights)
#pragma unroll
      for (int x = 0; x < V; ++x) y[x] *= weights[0];
    for (int s = 1; s < update.terms; ++s) {
      float more[V];
      load_v<V>(more, up + s * update.stride + i);
      const float w = weights ? weights[s] : 1.f;
#pragma unroll
      for (int x = 0; x < V; ++x) y[x] = fmaf(w, more[x], y[x]);
    }
  };
  if (update.gain == nullptr) {
    share.each<V>([&](int, int i) {
      float x[V], y[V];
      load_v<V>(x, res + i);
      pending(i, y);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] += y[e];
      store_v<V>(u_s + i, x);
      if (write_back) store_v<V>(res + i, x);
    });
    return;
  }
  float sq = 0.f;
  share.each<V>([&](int, int i) {
    float y[V];
    pending(i, y);
#pragma unroll
    for (int e = 0; e < V; ++e) sq = fmaf(y[e], y[e], sq);
    store_v<V>(u_s + i, y);
  });
  const float inv = rsqrtf(block_sum(sq, scratch) / (float)hidden + update.eps);
  share.each<V>([&](int, int i) {
    float x[V], y[V], g[V];
    load_v<V>(x, res + i);
    load_v<V>(y, u_s + i);
    load_v<V>(g, update.gain + i);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = fmaf(y[e] * inv, g[e], x[e]);
    store_v<V>(u_s + i, x);
    if (write_back) store_v<V>(res + i, x);
  });
}

struct Conv {
  const float* w;          // [hidden][taps], the last tap the current token's
  int taps;
  float* history;          // per slot [taps - 1][hidden], oldest first, `history_stride` floats from slot to slot
  long long history_stride;
  const int* slots;
  const int* active;       // per request: 0 leaves its history as it is
  int max_slots;
};

constexpr int kNorm = 0, kPlain = 1, kStats = 2, kNormConv = 3;

// One block per row.  kNorm: the norm; kPlain: the row itself, rounded; kStats: only inv [rows][groups];
// kNormConv: the norm and the convolution of single tokens (row t is request t).
template <typename T, int V, int MODE>
__global__ void __launch_bounds__(kMaxWarps * 32)
group_norm_kernel(float* residual, Update update, const float* __restrict__ gain, T* out, float* __restrict__ inv_out,
                  const int* __restrict__ rows, Share share, float eps, Conv conv, int* err) {
  extern __shared__ __align__(16) float u_s[];     // the row, then the parts' inverses
  __shared__ float scratch[33], warp_s[kMaxWarps];
  const int hidden = share.part * share.groups;
  float* inv_s = u_s + ((hidden + 3) & ~3);
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, src = rows ? rows[r] : r;
  stream_row<V>(share, residual, update, src, rows == nullptr, u_s, scratch);
  T* dst = out + (size_t)r * hidden;
  if constexpr (MODE == kPlain) {
    share.each<V>([&](int, int i) {
      float x[V];
      load_v<V>(x, u_s + i);
      store_v<V>(dst + i, x);
    });
    return;
  }
  part_inverses<V>(share, u_s, inv_s, warp_s, eps);
  if constexpr (MODE == kStats) {
    for (int g = threadIdx.x; g < share.groups; g += blockDim.x) inv_out[(size_t)r * share.groups + g] = inv_s[g];
    return;
  }
  float* hist = nullptr;
  bool keep = false;
  if constexpr (MODE == kNormConv) {
    const int slot = conv.slots[r];
    if (slot < 0 || slot >= conv.max_slots) {
      if (threadIdx.x == 0) atomicOr(err, kErrBadRequest);
      return;
    }
    hist = conv.history + (size_t)slot * conv.history_stride;
    keep = conv.active[r] != 0;
  }
  share.each<V>([&](int g, int i) {
    float h[V], w[V];
    load_v<V>(h, u_s + i);
    load_v<V>(w, gain + i);
#pragma unroll
    for (int e = 0; e < V; ++e) h[e] = w[e] * (h[e] * inv_s[g]);
    if constexpr (MODE == kNormConv) {
      float acc[V] = {}, older[V];
      for (int j = 0; j < conv.taps - 1; ++j) {
        load_v<V>(older, hist + (size_t)j * hidden + i);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(conv.w[(size_t)(i + e) * conv.taps + j], older[e], acc[e]);
        if (keep && j > 0) store_v<V>(hist + (size_t)(j - 1) * hidden + i, older);
      }
      if (keep && conv.taps > 1) store_v<V>(hist + (size_t)(conv.taps - 2) * hidden + i, h);
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] += fmaf(conv.w[(size_t)(i + e) * conv.taps + conv.taps - 1], h[e], acc[e]);
    }
    store_v<V>(dst + i, h);
  });
}

// The same with the row in registers: P pieces of four elements a thread, every part on warps of its own; all loads of
// a thread are asked for together.  Rows whose parts are whole pieces and fit.
template <typename T, int P, int MODE>
__global__ void __launch_bounds__(512)
group_norm_pieces_kernel(float* residual, Update update, const float* __restrict__ gain, T* out, float* __restrict__ inv_out,
                         const int* __restrict__ rows, Share share, float eps, Conv conv, int* err) {
  __shared__ float scratch[33], warp_s[kMaxWarps];
  const int hidden = share.part * share.groups;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = warp / share.wpg;
  const int first = ((warp % share.wpg) * 32 + lane) * 4, step = share.wpg * 128;
  const int column = g * share.part + first;
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, src = rows ? rows[r] : r;
  float* res = residual + (size_t)src * hidden + column;
  float x[P][4], w[P][4];
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const bool in = first + p * step < share.part;
#pragma unroll
    for (int e = 0; e < 4; ++e) x[p][e] = w[p][e] = 0.f;
    if (in) {
      load_v<4>(x[p], res + p * step);
      if (MODE == kNorm || MODE == kNormConv) load_v<4>(w[p], gain + column + p * step);
    }
  }
  if (update.data != nullptr) {
    const float* up = update.data + (size_t)src * update.row_stride + column;
    const float* weights = update.weights ? update.weights + (size_t)src * update.terms : nullptr;
    const float w0 = weights ? weights[0] : 1.f;
    float y[P][4];
#pragma unroll
    for (int p = 0; p < P; ++p) {
#pragma unroll
      for (int e = 0; e < 4; ++e) y[p][e] = 0.f;
      if (first + p * step < share.part) load_v<4>(y[p], up + p * step);
      if (weights)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[p][e] *= w0;
    }
    for (int s = 1; s < update.terms; ++s) {
      const float ws = weights ? weights[s] : 1.f;
#pragma unroll
      for (int p = 0; p < P; ++p) {
        if (first + p * step >= share.part) continue;
        float more[4];
        load_v<4>(more, up + s * update.stride + p * step);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[p][e] = fmaf(ws, more[e], y[p][e]);
      }
    }
    if (update.gain == nullptr) {
#pragma unroll
      for (int p = 0; p < P; ++p)
#pragma unroll
        for (int e = 0; e < 4; ++e) x[p][e] += y[p][e];
    } else {
      float gy[P][4], sq = 0.f;
#pragma unroll
      for (int p = 0; p < P; ++p) {
#pragma unroll
        for (int e = 0; e < 4; ++e) gy[p][e] = 0.f;
        if (first + p * step < share.part) load_v<4>(gy[p], update.gain + column + p * step);
#pragma unroll
        for (int e = 0; e < 4; ++e) sq = fmaf(y[p][e], y[p][e], sq);
      }
      const float inv = rsqrtf(block_sum(sq, scratch) / (float)hidden + update.eps);
#pragma unroll
      for (int p = 0; p < P; ++p)
#pragma unroll
        for (int e = 0; e < 4; ++e) x[p][e] = fmaf(y[p][e] * inv, gy[p][e], x[p][e]);
    }
    if (rows == nullptr)
#pragma unroll
      for (int p = 0; p < P; ++p)
        if (first + p * step < share.part) store_v<4>(res + p * step, x[p]);
  }
  T* dst = out + (size_t)r * hidden + column;
  if constexpr (MODE == kPlain) {
#pragma unroll
    for (int p = 0; p < P; ++p)
      if (first + p * step < share.part) store_v<4>(dst + p * step, x[p]);
    return;
  }
  float sq = 0.f;
#pragma unroll
  for (int p = 0; p < P; ++p)
#pragma unroll
    for (int e = 0; e < 4; ++e) sq = fmaf(x[p][e], x[p][e], sq);
  sq = warp_sum(sq);
  if (share.wpg > 1) {
    if (lane == 0) warp_s[warp] = sq;
    __syncthreads();
    sq = 0.f;
    for (int k = 0; k < share.wpg; ++k) sq += warp_s[g * share.wpg + k];
  }
  const float inv = rsqrtf(sq / (float)share.part + eps);
  if constexpr (MODE == kStats) {
    if (lane == 0 && warp % share.wpg == 0) inv_out[(size_t)r * share.groups + g] = inv;
    return;
  }
  float* hist = nullptr;
  bool keep = false;
  if constexpr (MODE == kNormConv) {
    const int slot = conv.slots[r];
    if (slot < 0 || slot >= conv.max_slots) {
      if (threadIdx.x == 0) atomicOr(err, kErrBadRequest);
      return;
    }
    hist = conv.history + (size_t)slot * conv.history_stride + column;
    keep = conv.active[r] != 0;
  }
#pragma unroll
  for (int p = 0; p < P; ++p) {
    if (first + p * step >= share.part) continue;
    float h[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = w[p][e] * (x[p][e] * inv);
    if constexpr (MODE == kNormConv) {
      const float* f = conv.w + (size_t)(column + p * step) * conv.taps;
      float acc[4] = {}, older[4];
      for (int j = 0; j < conv.taps - 1; ++j) {
        load_v<4>(older, hist + (size_t)j * hidden + p * step);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] = fmaf(f[e * conv.taps + j], older[e], acc[e]);
        if (keep && j > 0) store_v<4>(hist + (size_t)(j - 1) * hidden + p * step, older);
      }
      if (keep && conv.taps > 1) store_v<4>(hist + (size_t)(conv.taps - 2) * hidden + p * step, h);
#pragma unroll
      for (int e = 0; e < 4; ++e) h[e] += fmaf(f[e * conv.taps + conv.taps - 1], h[e], acc[e]);
    }
    store_v<4>(dst + p * step, h);
  }
}

// h of token row t at channel i from the stream and the row's statistics.
template <int V>
__device__ __forceinline__ void normed(float (&h)[V], const float* __restrict__ stream, const float* __restrict__ inv,
                                       const float (&gain)[V], int t, int i, int g, int hidden, int groups) {
  load_v<V>(h, stream + (size_t)t * hidden + i);
  const float s = inv[(size_t)t * groups + g];
#pragma unroll
  for (int e = 0; e < V; ++e) h[e] = gain[e] * (h[e] * s);
}

// grid (runs of kConvRun tokens, channel blocks): a thread keeps its channels' taps in registers and walks a run.
constexpr int kConvRun = 8, kConvThreads = 128;
template <typename T, int V, int TAPS>     // TAPS 0: any number
__global__ void __launch_bounds__(kConvThreads)
norm_conv_kernel(const float* __restrict__ stream, const float* __restrict__ inv, const float* __restrict__ gain,
                 T* __restrict__ out, const int* __restrict__ query_start, const int* __restrict__ request_of_token,
                 int tokens, int hidden, int groups, Conv conv, int* err) {
  pdl_wait();
  pdl_trigger();
  const int i = (blockIdx.y * kConvThreads + threadIdx.x) * V;
  if (i >= hidden) return;
  const int taps = TAPS ? TAPS : conv.taps;
  const int g = i / (hidden / groups);
  float gv[V], w[V][TAPS ? TAPS : 1];
  load_v<V>(gv, gain + i);
  if constexpr (TAPS > 0)
#pragma unroll
    for (int e = 0; e < V; ++e)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[e][j] = conv.w[(size_t)(i + e) * TAPS + j];
  const int t0 = blockIdx.x * kConvRun, t1 = min(t0 + kConvRun, tokens);
  float window[TAPS ? TAPS : 1][V];      // h of the request's last TAPS tokens
  int held = -1;                         // the request they belong to
  for (int t = t0; t < t1; ++t) {
    const int request = request_of_token[t], begin = query_start[request];
    const int slot = conv.slots[request];
    if (slot < 0 || slot >= conv.max_slots) {
      atomicOr(err, kErrBadRequest);
      return;
    }
    const float* hist = conv.history + (size_t)slot * conv.history_stride;
    auto fetch = [&](float (&h)[V], int src) {       // h of the request's token `src` of this step (< 0: an earlier one)
      if (src >= 0) normed<V>(h, stream, inv, gv, begin + src, i, g, hidden, groups);
      else load_v<V>(h, hist + (size_t)(taps - 1 + src) * hidden + i);
    };
    float acc[V] = {}, h[V];
    if constexpr (TAPS > 0) {
      if (request != held) {             // the run's first token, or another request's: fill the window
        held = request;
#pragma unroll
        for (int j = 1; j < TAPS; ++j) fetch(window[j], t - begin - (TAPS - j));
      }
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) window[j][e] = window[j + 1][e];
      fetch(window[TAPS - 1], t - begin);
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(w[e][j], window[j][e], acc[e]);
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] = window[TAPS - 1][e] + acc[e];
    } else {
      for (int j = 0; j < taps; ++j) {
        fetch(h, t - begin - (taps - 1 - j));
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(conv.w[(size_t)(i + e) * taps + j], h[e], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] += acc[e];       // the last tap read the token's own row
    }
    store_v<V>(out + (size_t)t * hidden + i, h);
  }
}

// The history after the step: h of the request's last taps - 1 tokens.  grid (requests, channel blocks).
template <int V>
__global__ void __launch_bounds__(kConvThreads)
norm_conv_keep_kernel(const float* __restrict__ stream, const float* __restrict__ inv, const float* __restrict__ gain,
                      const int* __restrict__ query_start, int hidden, int groups, Conv conv) {
  pdl_wait();
  pdl_trigger();
  const int request = blockIdx.x, i = (blockIdx.y * kConvThreads + threadIdx.x) * V;
  if (i >= hidden || !conv.active[request]) return;
  const int slot = conv.slots[request];
  if (slot < 0 || slot >= conv.max_slots) return;
  const int begin = query_start[request], count = query_start[request + 1] - begin, g = i / (hidden / groups);
  float* hist = conv.history + (size_t)slot * conv.history_stride;
  float gv[V], h[V];
  load_v<V>(gv, gain + i);
  // oldest first: an entry is read (from a later place) before its place is written
  for (int j = 0; j < conv.taps - 1; ++j) {
    const int src = count - (conv.taps - 1) + j;
    if (src >= 0) normed<V>(h, stream, inv, gv, begin + src, i, g, hidden, groups);
    else load_v<V>(h, hist + (size_t)(conv.taps - 1 + src) * hidden + i);
    store_v<V>(hist + (size_t)j * hidden + i, h);
  }
}

// One block per token: u = y * silu(z), each of the parts by its own root mean square, times gain.
template <typename T, int V>
__global__ void __launch_bounds__(kMaxWarps * 32)
gated_group_norm_kernel(const float* __restrict__ y, int y_stride, const float* __restrict__ z, int z_stride,
                        const float* __restrict__ gain, T* __restrict__ out, int out_stride, Share share, float eps) {
  extern __shared__ __align__(16) float u_s[];
  __shared__ float warp_s[kMaxWarps];
  float* inv_s = u_s + ((share.part * share.groups + 3) & ~3);
  pdl_wait();
  pdl_trigger();
  const float* yr = y + (size_t)blockIdx.x * y_stride;
  const float* zr = z + (size_t)blockIdx.x * z_stride;
  share.each<V>([&](int, int i) {
    float a[V], b[V];
    load_v<V>(a, yr + i);
    load_v<V>(b, zr + i);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] *= silu_f(b[e]);
    store_v<V>(u_s + i, a);
  });
  part_inverses<V>(share, u_s, inv_s, warp_s, eps);
  T* dst = out + (size_t)blockIdx.x * out_stride;
  share.each<V>([&](int g, int i) {
    float a[V], w[V];
    load_v<V>(a, u_s + i);
    load_v<V>(w, gain + i);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] = w[e] * (a[e] * inv_s[g]);
    store_v<V>(dst + i, a);
  });
}

// out[t][c] = gelu_tanh(z[t][c]) * table[ids[t]][column + c]
template <typename T>
__global__ void side_gate_kernel(const float* __restrict__ z, const int* __restrict__ ids, const T* __restrict__ table,
                                 int table_width, int vocab, int column, T* __restrict__ out, int tokens, int dim, int* err) {
  pdl_wait();
  pdl_trigger();
  const size_t total = (size_t)tokens * dim;
  for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
    const int t = (int)(e / dim), c = (int)(e % dim);
    int id = ids[t];
    if (id < 0 || id >= vocab) {
      atomicOr(err, kErrBadToken);
      id = 0;
    }
    out[e] = from_float<T>(gelu_tanh_f(z[e]) * to_float(table[(size_t)id * table_width + column + c]));
  }
}

}  // namespace cie

using namespace cie;

#define DISPATCH_DTYPE(dtype, name, ...)                                   \
  if (dtype == kFloat32) { using T = float; __VA_ARGS__ }                 \
  else if (dtype == kBFloat16) { using T = __nv_bfloat16; __VA_ARGS__ }   \
  else CIE_FAIL("%s: unknown element type code %d", name, dtype);

// Warps for a row of `groups` parts: about eight elements a thread.
static int share_row(Share* share, int hidden, int groups) {
  share->groups = groups;
  share->part = hidden / groups;
  if (groups > 16) {
    share->wpg = 1;
    return 32 * (groups < 16 ? groups : 16);
  }
  int wpg = (hidden + 8 * 32 * groups - 1) / (8 * 32 * groups);
  const int most = kMaxWarps / groups;
  share->wpg = wpg < 1 ? 1 : (wpg > most ? most : wpg);
  return 32 * share->wpg * groups;
}

template <typename K>
static int allow_shared(K kernel, size_t bytes, const char* name) {
  if (bytes > 200 * 1024) CIE_FAIL("%s: a row of %zu bytes does not fit shared memory", name, bytes);
  if (bytes > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess)
    CIE_FAIL("%s: cannot reserve %zu bytes of shared memory", name, bytes);
  return 0;
}

static bool aligned16(const void* a, const void* b, const void* c, const void* d) {
  return ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c) |
           reinterpret_cast<uintptr_t>(d)) & 15) == 0;
}

// Pieces a thread of the kernel that keeps rows in registers would hold (0: not its kind).
static int pieces_of(const Share& share, int threads) {
  if (threads != 32 * share.wpg * share.groups || threads > 512) return 0;
  const int pieces = (share.part + share.wpg * 128 - 1) / (share.wpg * 128);
  return pieces <= 4 ? pieces : 0;
}
#define CIE_PIECES(name, P, MODE, count, out, inv, rows, conv, err)                                                  \
  CIE_LAUNCH(name, (group_norm_pieces_kernel<T, P, MODE>), dim3(count), dim3(threads), 0, (cudaStream_t)stream,      \
             residual, up, gain, (T*)(out), (float*)(inv), (const int*)(rows), share, eps, conv, (int*)(err))

extern "C" int cie_norm_conv_max_taps() { return kMaxTaps; }

// mode: 0 norm, 1 the rows themselves (gain unused).  out_dtype: float32 or bfloat16 (`out` may be the stream
// itself in float32: a row is read whole before it is written).
extern "C" int cie_group_norm(float* residual, const float* update, int terms, long long stride, long long row_stride,
                              const float* weights, const float* update_gain, float update_eps, const float* gain, void* out, const int* rows, int count, int hidden,
                              int groups, float eps, int mode, int out_dtype, void* stream) {
  if (count <= 0) return 0;
  if (groups < 1 || hidden < 1 || hidden % groups) CIE_FAIL("group_norm: a row of %d in %d parts", hidden, groups);
  if (update && (terms < 1 || terms > kMaxTerms)) CIE_FAIL("group_norm: 1..%d float32 terms, got %d", kMaxTerms, terms);
  if (mode != kNorm && mode != kPlain) CIE_FAIL("group_norm: unknown mode %d", mode);
  Share share;
  const int threads = share_row(&share, hidden, groups);
  const Update up{update, terms, (size_t)stride, (size_t)row_stride, weights, update_gain, update_eps};
  const size_t smem = (size_t)(((hidden + 3) & ~3) + groups) * sizeof(float);
  const bool wide = share.part % 4 == 0 && stride % 4 == 0 && row_stride % 4 == 0 && aligned16(residual, update, gain, out) && aligned16(update_gain, 0, 0, 0);
#define CIE_GROUP_NORM(V, MODE)                                                                                     \
  do {                                                                                                               \
    if (V == 4 && pieces_of(share, threads) == 1) { CIE_PIECES("group_norm", 1, MODE, count, out, nullptr, rows, Conv{}, nullptr); break; } \
    if (V == 4 && pieces_of(share, threads) == 2) { CIE_PIECES("group_norm", 2, MODE, count, out, nullptr, rows, Conv{}, nullptr); break; } \
    if (V == 4 && pieces_of(share, threads) > 0) { CIE_PIECES("group_norm", 4, MODE, count, out, nullptr, rows, Conv{}, nullptr); break; } \
    if (allow_shared(group_norm_kernel<T, V, MODE>, smem, "group_norm")) return 1;                                   \
    CIE_LAUNCH("group_norm", (group_norm_kernel<T, V, MODE>), dim3(count), dim3(threads), smem, (cudaStream_t)stream, \
               residual, up, gain, (T*)out, (float*)nullptr, rows, share, eps, Conv{}, (int*)nullptr);               \
  } while (0)
  DISPATCH_DTYPE(out_dtype, "group_norm", {
    if (mode == kNorm) { if (wide) CIE_GROUP_NORM(4, kNorm); else CIE_GROUP_NORM(1, kNorm); }
    else { if (wide) CIE_GROUP_NORM(4, kPlain); else CIE_GROUP_NORM(1, kPlain); }
  })
#undef CIE_GROUP_NORM
  return 0;
}

// singles: every request brings one token (row t is request t).  inv: float32 scratch [tokens][groups], used otherwise.
extern "C" int cie_group_norm_conv(float* residual, const float* update, int terms, long long stride, long long row_stride,
                                   const float* weights, const float* update_gain, float update_eps, const float* gain, void* out, float* inv,
                                   const float* w, int taps, float* history, long long history_stride,
                                   const int* query_start, const int* request_of_token, const int* slots,
                                   const int* request_active, int tokens, int requests, int max_slots, int hidden,
                                   int groups, float eps, int singles, int dtype, int* err, void* stream) {
  if (tokens <= 0) return 0;
  if (groups < 1 || hidden < 1 || hidden % groups) CIE_FAIL("group_norm_conv: a row of %d in %d parts", hidden, groups);
  if (update && (terms < 1 || terms > kMaxTerms)) CIE_FAIL("group_norm_conv: 1..%d float32 terms, got %d", kMaxTerms, terms);
  if (taps < 1 || taps > kMaxTaps) CIE_FAIL("group_norm_conv: %d taps (1..%d)", taps, kMaxTaps);
  if (singles && tokens != requests) CIE_FAIL("group_norm_conv: %d tokens of %d requests are not single tokens", tokens, requests);
  Share share;
  const int threads = share_row(&share, hidden, groups);
  const Update up{update, terms, (size_t)stride, (size_t)row_stride, weights, update_gain, update_eps};
  const Conv conv{w, taps, history, history_stride, slots, request_active, max_slots};
  const size_t smem = (size_t)(((hidden + 3) & ~3) + groups) * sizeof(float);
  const bool wide = share.part % 4 == 0 && stride % 4 == 0 && row_stride % 4 == 0 && history_stride % 4 == 0 && aligned16(residual, update, gain, out) &&
                    aligned16(update_gain, history, 0, 0);
#define CIE_CONV_STEP(V)                                                                                             \
  do {                                                                                                               \
    const int pieces = V == 4 ? pieces_of(share, threads) : 0;                                                       \
    if (singles && pieces) {                                                                                         \
      if (pieces == 1) CIE_PIECES("group_norm_conv", 1, kNormConv, tokens, out, nullptr, nullptr, conv, err);        \
      else if (pieces == 2) CIE_PIECES("group_norm_conv", 2, kNormConv, tokens, out, nullptr, nullptr, conv, err);   \
      else CIE_PIECES("group_norm_conv", 4, kNormConv, tokens, out, nullptr, nullptr, conv, err);                    \
      return 0;                                                                                                      \
    }                                                                                                                \
    if (singles) {                                                                                                   \
      if (allow_shared(group_norm_kernel<T, V, kNormConv>, smem, "group_norm_conv")) return 1;                       \
      CIE_LAUNCH("group_norm_conv", (group_norm_kernel<T, V, kNormConv>), dim3(tokens), dim3(threads), smem,         \
                 (cudaStream_t)stream, residual, up, gain, (T*)out, (float*)nullptr, (const int*)nullptr, share, eps, \
                 conv, err);                                                                                         \
      return 0;                                                                                                      \
    }                                                                                                                \
    if (pieces == 1) CIE_PIECES("group_norm_stats", 1, kStats, tokens, nullptr, inv, nullptr, conv, err);            \
    else if (pieces == 2) CIE_PIECES("group_norm_stats", 2, kStats, tokens, nullptr, inv, nullptr, conv, err);       \
    else if (pieces) CIE_PIECES("group_norm_stats", 4, kStats, tokens, nullptr, inv, nullptr, conv, err);            \
    else {                                                                                                           \
      if (allow_shared(group_norm_kernel<T, V, kStats>, smem, "group_norm_conv")) return 1;                          \
      CIE_LAUNCH("group_norm_stats", (group_norm_kernel<T, V, kStats>), dim3(tokens), dim3(threads), smem,           \
                 (cudaStream_t)stream, residual, up, gain, (T*)nullptr, inv, (const int*)nullptr, share, eps, conv,  \
                 err);                                                                                               \
    }                                                                                                                \
    const int blocks = (hidden + V * kConvThreads - 1) / (V * kConvThreads);                                         \
    const dim3 grid((tokens + kConvRun - 1) / kConvRun, blocks);                                                     \
    if (taps == 2) CIE_CONV_RUN(V, 2); else if (taps == 3) CIE_CONV_RUN(V, 3);                                       \
    else if (taps == 4) CIE_CONV_RUN(V, 4); else CIE_CONV_RUN(V, 0);                                                 \
    if (taps > 1)                                                                                                    \
      CIE_LAUNCH("norm_conv_keep", norm_conv_keep_kernel<V>, dim3(requests, blocks), dim3(kConvThreads), 0,          \
                 (cudaStream_t)stream, (const float*)residual, (const float*)inv, gain, query_start, hidden, groups, conv); \
  } while (0)
#define CIE_CONV_RUN(V, N)                                                                                           \
  CIE_LAUNCH("norm_conv", (norm_conv_kernel<T, V, N>), grid, dim3(kConvThreads), 0, (cudaStream_t)stream,            \
             (const float*)residual, (const float*)inv, gain, (T*)out, query_start, request_of_token, tokens, hidden, \
             groups, conv, err)
  DISPATCH_DTYPE(dtype, "group_norm_conv", {
    if (wide) CIE_CONV_STEP(4);
    else CIE_CONV_STEP(1);
  })
#undef CIE_CONV_RUN
#undef CIE_CONV_STEP
  return 0;
}

extern "C" int cie_gated_group_norm(const float* y, int y_stride, const float* z, int z_stride, const float* gain, void* out,
                                    int out_stride, int tokens, int width, int groups, float eps, int dtype, void* stream) {
  if (tokens <= 0) return 0;
  if (groups < 1 || width < 1 || width % groups) CIE_FAIL("gated_group_norm: a row of %d in %d parts", width, groups);
  Share share;
  const int threads = share_row(&share, width, groups);
  const size_t smem = (size_t)(((width + 3) & ~3) + groups) * sizeof(float);
  const bool wide = share.part % 4 == 0 && y_stride % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0 && aligned16(y, z, gain, out);
#define CIE_GATED(V)                                                                                                 \
  do {                                                                                                               \
    if (allow_shared(gated_group_norm_kernel<T, V>, smem, "gated_group_norm")) return 1;                             \
    CIE_LAUNCH("gated_group_norm", (gated_group_norm_kernel<T, V>), dim3(tokens), dim3(threads), smem,               \
               (cudaStream_t)stream, y, y_stride, z, z_stride, gain, (T*)out, out_stride, share, eps);               \
  } while (0)
  DISPATCH_DTYPE(dtype, "gated_group_norm", {
    if (wide) CIE_GATED(4);
    else CIE_GATED(1);
  })
#undef CIE_GATED
  return 0;
}

extern "C" int cie_side_gate(const float* z, const int* ids, const void* table, int table_width, int vocab, int column,
                             void* out, int tokens, int dim, int dtype, int* err, void* stream) {
  if (tokens <= 0 || dim <= 0) return 0;
  if (column < 0 || column + dim > table_width) CIE_FAIL("side_gate: columns %d.. of %d do not lie in a row of %d", column, dim, table_width);
  const size_t total = (size_t)tokens * dim;
  int blocks = (int)((total + 255) / 256);
  if (blocks > 148 * 16) blocks = 148 * 16;
  DISPATCH_DTYPE(dtype, "side_gate", {
    CIE_LAUNCH("side_gate", side_gate_kernel<T>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, z, ids,
               (const T*)table, table_width, vocab, column, (T*)out, tokens, dim, err);
  })
  return 0;
}

// One step of a residual stream whose sublayers are normalised on their OUTPUT, whose layers may read an average over
// everything earlier layers left, and whose mixers may read every row moved towards the row before it:
//
//   advance   per row t of the float32 stream
//               y    the pending update: float32 terms (a sublayer's result, or a token's expert outputs, each
//                    optionally times a weight of its own) plus, optionally, one more result (`extra`)
//               r    = base + y, or base + gain * rms_norm(y), or base + gain * layer_norm(y)
//                    (kept in the row's history if `keep` is given)
//               x    = r, or sum_j share[j] * history_j + share[states] * r   (`share`)
//                    (written to the stream if `stream` is given)
//             and then out = x rounded to the activation type, or a layer norm of x, or (`kShift`)
//               out  = x + (x' - x) * shift   with x' the x of the request's token before it
//   shift_portions   the last line for rows whose x' belongs to the same step, and the state left behind
//
// A request's x of its last token is its state (zeros before the first).  `advance` itself finishes the first row of
// every request (it reads the state) and, where that is the request's only row, leaves the new state: a step of
// single tokens is one launch.  All sums, statistics and the stream are float32; a result is rounded once.  A row's
// result depends on its own request's rows alone.
#include "common.cuh"

CIE_DEFINE_LAST_ERROR()

namespace cie {

constexpr int kMaxTerms = 64;      // float32 terms of a pending update
constexpr int kPlain = 0, kCentred = 2;                     // how the pending update is normalised (1: RMS)
constexpr int kRounded = 0, kShift = 1, kNormed = 2;        // what `out` gets

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

struct Pending {
  const float* terms;      // term s of row t at t * row_stride + s * stride; nullptr: nothing pending
  int count;
  size_t stride, row_stride;
  const float* weights;    // not null: term s of row t is multiplied by weights[t * count + s]
  const float* extra;      // not null: `extras` more terms (a result, whole or cut), term s of row t at t * hidden + s * extra_stride
  int extras;
  size_t extra_stride;
  const float* gain;       // [hidden], for kRms and kCentred
  float eps;
  int kind;
};

struct Depth {
  const float* base;       // row t at t * base_stride
  size_t base_stride;
  const float* history;    // state j of row t at t * history_stride + j * hidden
  size_t history_stride;
  int states;              // earlier states that the average reads
  const float* share;      // [states + 1] or nullptr: no average
  float* keep;             // row t at t * keep_stride, or nullptr
  size_t keep_stride;
  float* stream;           // [rows][hidden] or nullptr
};

struct Shift {
  const float* share;      // [hidden]
  float* state;            // per slot [hidden], `stride` floats from slot to slot
  long long stride;
  const int* query_start;
  const int* request_of_token;
  const int* slots;
  const int* active;       // per request: 0 leaves its state as it is
  int max_slots;
};

// P pieces of V elements a thread; one block per row.
template <typename T, int V, int P, int OUT>
__global__ void __launch_bounds__(P > 8 ? 1024 : 512)
advance_kernel(Pending pending, Depth depth, T* __restrict__ out, const int* __restrict__ rows, Shift shift,
               const float* __restrict__ out_gain, float out_eps, int hidden, int* err) {
  __shared__ float scratch[33];
  const int first = threadIdx.x * V, step = blockDim.x * V;
  auto in = [&](int p) { return first + p * step < hidden; };
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, t = rows ? rows[r] : r;
  float x[P][V], acc[P][V];
  const float* base = depth.base + (size_t)t * depth.base_stride + first;
#pragma unroll
  for (int p = 0; p < P; ++p) {
#pragma unroll
    for (int e = 0; e < V; ++e) x[p][e] = acc[p][e] = 0.f;
    if (in(p)) load_v<V>(x[p], base + p * step);
  }
  if (depth.share) {       // what the average takes of earlier states does not wait for the pending update
    const float* history = depth.history + (size_t)t * depth.history_stride + first;
#pragma unroll 4
    for (int j = 0; j < depth.states; ++j) {
      const float share = depth.share[j];
#pragma unroll
      for (int p = 0; p < P; ++p) {
        if (!in(p)) continue;
        float h[V];
        load_v<V>(h, history + (size_t)j * hidden + p * step);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[p][e] = fmaf(share, h[e], acc[p][e]);
      }
    }
  }
  if (pending.terms) {
    const float* terms = pending.terms + (size_t)t * pending.row_stride + first;
    const float* weights = pending.weights ? pending.weights + (size_t)t * pending.count : nullptr;
    float y[P][V];
#pragma unroll
    for (int p = 0; p < P; ++p)
#pragma unroll
      for (int e = 0; e < V; ++e) y[p][e] = 0.f;
#pragma unroll 4
    for (int s = 0; s < pending.count; ++s) {
      const float w = weights ? weights[s] : 1.f;
#pragma unroll
      for (int p = 0; p < P; ++p) {
        if (!in(p)) continue;
        float more[V];
        load_v<V>(more, terms + s * pending.stride + p * step);
#pragma unroll
        for (int e = 0; e < V; ++e) y[p][e] = fmaf(w, more[e], y[p][e]);
      }
    }
    if (pending.extra) {
      const float* extra = pending.extra + (size_t)t * hidden + first;
#pragma unroll
      for (int p = 0; p < P; ++p) {
        if (!in(p)) continue;
        for (int s = 0; s < pending.extras; ++s) {
          float more[V];
          load_v<V>(more, extra + s * pending.extra_stride + p * step);
#pragma unroll
          for (int e = 0; e < V; ++e) y[p][e] += more[e];
        }
      }
    }
    if (pending.kind == kPlain) {
#pragma unroll
      for (int p = 0; p < P; ++p)
#pragma unroll
        for (int e = 0; e < V; ++e) x[p][e] += y[p][e];
    } else {
      float mean = 0.f;
      if (pending.kind == kCentred) {
        float sum = 0.f;
#pragma unroll
        for (int p = 0; p < P; ++p)
#pragma unroll
          for (int e = 0; e < V; ++e) sum += y[p][e];
        mean = block_sum(sum, scratch) / (float)hidden;
      }
      float sq = 0.f;
#pragma unroll
      for (int p = 0; p < P; ++p) {
        if (!in(p)) continue;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          y[p][e] -= mean;
          sq = fmaf(y[p][e], y[p][e], sq);
        }
      }
      const float inv = rsqrtf(block_sum(sq, scratch) / (float)hidden + pending.eps);
#pragma unroll
      for (int p = 0; p < P; ++p) {
        if (!in(p)) continue;
        float g[V];
        load_v<V>(g, pending.gain + first + p * step);
#pragma unroll
        for (int e = 0; e < V; ++e) x[p][e] = fmaf(g[e], y[p][e] * inv, x[p][e]);
      }
    }
  }
  if (depth.keep) {
    float* keep = depth.keep + (size_t)t * depth.keep_stride + first;
#pragma unroll
    for (int p = 0; p < P; ++p)
      if (in(p)) store_v<V>(keep + p * step, x[p]);
  }
  if (depth.share) {
    const float share = depth.share[depth.states];
#pragma unroll
    for (int p = 0; p < P; ++p)
#pragma unroll
      for (int e = 0; e < V; ++e) x[p][e] = fmaf(share, x[p][e], acc[p][e]);
  }
  if (depth.stream) {
    float* stream = depth.stream + (size_t)t * hidden + first;
#pragma unroll
    for (int p = 0; p < P; ++p)
      if (in(p)) store_v<V>(stream + p * step, x[p]);
  }
  T* dst = out + (size_t)r * hidden + first;
  if constexpr (OUT == kRounded) {
#pragma unroll
    for (int p = 0; p < P; ++p)
      if (in(p)) store_v<V>(dst + p * step, x[p]);
  } else if constexpr (OUT == kShift) {
    const int request = shift.request_of_token[t];
    if (shift.query_start[request] != t) return;            // its x' is a row of this step: shift_portions
    const int slot = shift.slots[request];
    if (slot < 0 || slot >= shift.max_slots) {
      if (threadIdx.x == 0) atomicOr(err, kErrBadRequest);
      return;
    }
    const bool leave = shift.query_start[request + 1] == t + 1 && shift.active[request] != 0;
    float* state = shift.state + (size_t)slot * shift.stride + first;
#pragma unroll
    for (int p = 0; p < P; ++p) {
      if (!in(p)) continue;
      float before[V], share[V], h[V];
      load_v<V>(before, state + p * step);
      load_v<V>(share, shift.share + first + p * step);
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] = fmaf(before[e] - x[p][e], share[e], x[p][e]);
      store_v<V>(dst + p * step, h);
      if (leave) store_v<V>(state + p * step, x[p]);
    }
  } else {
    float sum = 0.f;
#pragma unroll
    for (int p = 0; p < P; ++p)
#pragma unroll
      for (int e = 0; e < V; ++e) sum += in(p) ? x[p][e] : 0.f;
    const float mean = block_sum(sum, scratch) / (float)hidden;
    float sq = 0.f;
#pragma unroll
    for (int p = 0; p < P; ++p) {
      if (!in(p)) continue;
#pragma unroll
      for (int e = 0; e < V; ++e) sq = fmaf(x[p][e] - mean, x[p][e] - mean, sq);
    }
    const float inv = rsqrtf(block_sum(sq, scratch) / (float)hidden + out_eps);
#pragma unroll
    for (int p = 0; p < P; ++p) {
      if (!in(p)) continue;
      float g[V], h[V];
      load_v<V>(g, out_gain + first + p * step);
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] = g[e] * ((x[p][e] - mean) * inv);
      store_v<V>(dst + p * step, h);
    }
  }
}

// grid (runs of kRun tokens, column blocks): a thread walks a run of rows of the stream with the row before in registers.
constexpr int kRun = 8, kRunThreads = 128;
template <typename T, int V>
__global__ void __launch_bounds__(kRunThreads)
shift_portions_kernel(const float* __restrict__ stream, T* __restrict__ out, Shift shift, int tokens, int hidden) {
  const int column = (blockIdx.y * kRunThreads + threadIdx.x) * V;
  pdl_wait();
  pdl_trigger();
  if (column >= hidden) return;
  const int t0 = blockIdx.x * kRun, t1 = min(t0 + kRun, tokens);
  float share[V], before[V] = {}, x[V];
  load_v<V>(share, shift.share + column);
  if (t0 > 0) load_v<V>(before, stream + (size_t)(t0 - 1) * hidden + column);
  int request = shift.request_of_token[t0], begin = shift.query_start[request], end = shift.query_start[request + 1];
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    if (t >= end) {
      request = shift.request_of_token[t];
      begin = shift.query_start[request];
      end = shift.query_start[request + 1];
    }
    load_v<V>(x, stream + (size_t)t * hidden + column);
    if (t != begin) {                  // a request's first row is finished already
      float h[V];
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] = fmaf(before[e] - x[e], share[e], x[e]);
      store_v<V>(out + (size_t)t * hidden + column, h);
      const int slot = shift.slots[request];
      if (t + 1 == end && shift.active[request] != 0 && slot >= 0 && slot < shift.max_slots)
        store_v<V>(shift.state + (size_t)slot * shift.stride + column, x);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) before[e] = x[e];
  }
}

}  // namespace cie

using namespace cie;

#define DISPATCH_DTYPE(dtype, name, ...)                                   \
  if (dtype == kFloat32) { using T = float; __VA_ARGS__ }                 \
  else if (dtype == kBFloat16) { using T = __nv_bfloat16; __VA_ARGS__ }   \
  else CIE_FAIL("%s: unknown element type code %d", name, dtype);

static bool aligned16(const void* a, const void* b, const void* c, const void* d) {
  return ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c) |
           reinterpret_cast<uintptr_t>(d)) & 15) == 0;
}

// The widest row: 16 pieces of one element for each of 1,024 threads.
extern "C" int cie_stream_step_max_width() { return 16 * 1024; }

// pending_kind: 0 plain, 1 RMS norm, 2 layer norm.  out_kind: 0 rounded rows, 1 shifted (singles: every request of the
// step brings one token), 2 layer norm with out_gain.  rows (or nullptr): which rows; then nothing but `out` may be
// asked for.
extern "C" int cie_stream_advance(const float* base, long long base_stride, const float* terms, int count,
                                  long long stride, long long row_stride, const float* weights, const float* extra,
                                  int extras, long long extra_stride, const float* gain, float eps, int pending_kind, const float* history,
                                  long long history_stride, int states, const float* share, float* keep,
                                  long long keep_stride, float* stream, void* out, int out_kind, const int* rows,
                                  int out_rows, int hidden, const float* shift_share, float* state, long long state_stride,
                                  const int* query_start, const int* request_of_token, const int* slots,
                                  const int* active, int max_slots, int singles, const float* out_gain, float out_eps,
                                  int dtype, int* err, void* cuda_stream) {
  if (out_rows <= 0) return 0;
  if (hidden < 1 || hidden > cie_stream_step_max_width()) CIE_FAIL("stream_advance: a row of %d elements (at most %d)", hidden, cie_stream_step_max_width());
  if (terms && (count < 1 || count > kMaxTerms)) CIE_FAIL("stream_advance: 1..%d float32 terms, got %d", kMaxTerms, count);
  if (extra && (extras < 1 || extras > kMaxTerms)) CIE_FAIL("stream_advance: 1..%d further terms, got %d", kMaxTerms, extras);
  if (pending_kind < 0 || pending_kind > 2 || out_kind < 0 || out_kind > 2) CIE_FAIL("stream_advance: kinds %d, %d", pending_kind, out_kind);
  if (terms && pending_kind != kPlain && !gain) CIE_FAIL("stream_advance: a normalised update needs its gain");
  if (rows && (keep || stream || out_kind == kShift)) CIE_FAIL("stream_advance: chosen rows are only read");
  if (out_kind == kShift && (!shift_share || !state)) CIE_FAIL("stream_advance: a shift needs its vector and state");
  if (out_kind == kShift && !singles && !stream && base_stride != hidden) CIE_FAIL("stream_advance: portions are shifted from the stream");
  if (out_kind == kNormed && !out_gain) CIE_FAIL("stream_advance: a norm needs its gain");
  const Pending pending{terms, count, (size_t)stride, (size_t)row_stride, weights, extra, extras, (size_t)extra_stride, gain, eps, pending_kind};
  const Depth depth{base, (size_t)base_stride, history, (size_t)history_stride, states, share, keep, (size_t)keep_stride, stream};
  const Shift shift{shift_share, state, state_stride, query_start, request_of_token, slots, active, max_slots};
  const bool wide = hidden % 4 == 0 && base_stride % 4 == 0 && stride % 4 == 0 && row_stride % 4 == 0 && extra_stride % 4 == 0 && history_stride % 4 == 0 &&
                    keep_stride % 4 == 0 && state_stride % 4 == 0 && aligned16(base, terms, extra, gain) &&
                    aligned16(history, keep, stream, out) && aligned16(shift_share, state, out_gain, nullptr);
  const int pieces = wide ? hidden / 4 : hidden;
  int per_thread = 1;
  while (per_thread < 8 && pieces > per_thread * 512) per_thread *= 2;
  if (pieces > per_thread * 512) per_thread = 16;
  const int threads = ((pieces + per_thread - 1) / per_thread + 31) / 32 * 32;
#define CIE_ADVANCE_P(V, P, OUT)                                                                                     \
  CIE_LAUNCH("stream_advance", (advance_kernel<T, V, P, OUT>), dim3(out_rows), dim3(threads), 0, (cudaStream_t)cuda_stream, \
             pending, depth, (T*)out, rows, shift, out_gain, out_eps, hidden, err)
#define CIE_ADVANCE_V(V, OUT)                                                                                        \
  do {                                                                                                               \
    if (per_thread == 1) CIE_ADVANCE_P(V, 1, OUT);                                                                   \
    else if (per_thread == 2) CIE_ADVANCE_P(V, 2, OUT);                                                              \
    else if (per_thread == 4) CIE_ADVANCE_P(V, 4, OUT);                                                              \
    else if (per_thread == 8 || V == 4) CIE_ADVANCE_P(V, 8, OUT);                                                    \
    else CIE_ADVANCE_P(1, 16, OUT);                                                                                  \
  } while (0)
#define CIE_ADVANCE(OUT)                                                                                             \
  do { if (wide) CIE_ADVANCE_V(4, OUT); else CIE_ADVANCE_V(1, OUT); } while (0)
  DISPATCH_DTYPE(dtype, "stream_advance", {
    if (out_kind == kRounded) CIE_ADVANCE(kRounded);
    else if (out_kind == kShift) CIE_ADVANCE(kShift);
    else CIE_ADVANCE(kNormed);
    if (out_kind == kShift && !singles) {
      const float* rows_of = stream ? stream : base;       // without a stream to write, x is the base itself
      const int span = kRunThreads * (wide ? 4 : 1);
      const dim3 grid((out_rows + kRun - 1) / kRun, (hidden + span - 1) / span);
      if (wide)
        CIE_LAUNCH("shift_portions", (shift_portions_kernel<T, 4>), grid, dim3(kRunThreads), 0, (cudaStream_t)cuda_stream,
                   rows_of, (T*)out, shift, out_rows, hidden);
      else
        CIE_LAUNCH("shift_portions", (shift_portions_kernel<T, 1>), grid, dim3(kRunThreads), 0, (cudaStream_t)cuda_stream,
                   rows_of, (T*)out, shift, out_rows, hidden);
    }
  })
#undef CIE_ADVANCE
#undef CIE_ADVANCE_V
#undef CIE_ADVANCE_P
  return 0;
}

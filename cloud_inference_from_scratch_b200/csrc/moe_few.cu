// The products of routed experts for a step of few (token, expert) pairs, a decode step: what they cost is one pass over
// the chosen experts' weights, so a warp streams whole weight rows (16-byte loads, many in flight) and multiplies them
// with the rows of the expert's pairs on the CUDA cores, float32 sums.  No plan and no gathered rows: a CTA belongs to
// one expert and finds that expert's pairs in the choices itself; one whose expert nobody chose leaves at once.
//
//   gate_up  W = [experts][2F][H], gate and up rows of an expert interleaved in blocks of 16 (moe_tcgen05.cu);
//            act[pair][channel], bfloat16, with the gated activation of glu.cuh
//   down     W = [experts][H][F]; rows[pair][column], float32
//
// A pair's result depends on the pair alone: every sum runs over k in one fixed order.
#include "common.cuh"
#include "glu.cuh"

CIE_DEFINE_LAST_ERROR()

namespace cie {

using bf16 = __nv_bfloat16;
constexpr int kFewPairs = 64;        // most pairs of a step
constexpr int kWarps = 8;
constexpr int kRows = 4;             // weight rows of a warp
constexpr int kTokens = 4;           // pairs of a pass over the weights

__device__ __forceinline__ float2 unpack(uint32_t v) {
  return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
}

// grid (blocks of 32 weight rows, experts).  x: gate_up: token rows [tokens][k], the row of pair p is x[p / top]; down: rows
// by pair [pairs][k].  n: weight rows of an expert (2F or H).
template <bool kGateUp>
__global__ void __launch_bounds__(kWarps * 32)
moe_few_kernel(const bf16* __restrict__ x, const bf16* __restrict__ w, void* __restrict__ out, const int* __restrict__ ids,
               int pairs, int top, int n, int k, GluAct act) {
  extern __shared__ __align__(16) uint4 x_s[];         // [kTokens][k / 8]
  __shared__ int list_s[kFewPairs], count_s;
  const int expert = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  if (warp == 0) {                                      // this expert's pairs, ascending
    int count = 0;
    for (int p0 = 0; p0 < pairs; p0 += 32) {
      const bool mine = p0 + lane < pairs && ids[p0 + lane] == expert;
      const unsigned votes = __ballot_sync(0xffffffffu, mine);
      if (mine) list_s[count + __popc(votes & ((1u << lane) - 1u))] = p0 + lane;
      count += __popc(votes);
    }
    if (lane == 0) count_s = count;
  }
  __syncthreads();
  const int count = count_s, pieces = k / 8;
  if (count == 0) return;
  int row[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i)
    row[i] = 32 * blockIdx.x + (kGateUp ? 2 * warp + (i & 1) + 16 * (i >> 1) : kRows * warp + i);
  const uint4* rows[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i)                       // a row beyond the last is read as the last and not stored
    rows[i] = reinterpret_cast<const uint4*>(w + ((size_t)expert * n + min(row[i], n - 1)) * k);
  for (int first = 0; first < count; first += kTokens) {
    const int here = min(kTokens, count - first);
    if (first > 0) __syncthreads();
    for (int e = threadIdx.x; e < kTokens * pieces; e += blockDim.x) {
      const int j = e / pieces, c = e - j * pieces;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (j < here) {
        const int pair = list_s[first + j];
        v = reinterpret_cast<const uint4*>(x + (size_t)(kGateUp ? pair / top : pair) * k)[c];
      }
      x_s[e] = v;
    }
    __syncthreads();
    float acc[kRows][kTokens];
#pragma unroll
    for (int i = 0; i < kRows; ++i)
#pragma unroll
      for (int j = 0; j < kTokens; ++j) acc[i][j] = 0.f;
    constexpr int kAhead = 4;                           // pieces of a row asked for together
    for (int c0 = lane; c0 < pieces; c0 += 32 * kAhead) {
      uint4 wv[kAhead][kRows];
#pragma unroll
      for (int u = 0; u < kAhead; ++u)
#pragma unroll
        for (int i = 0; i < kRows; ++i)
          wv[u][i] = c0 + 32 * u < pieces ? __ldg(rows[i] + c0 + 32 * u) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {
        if (c0 + 32 * u >= pieces) break;
#pragma unroll
        for (int j = 0; j < kTokens; ++j) {
          if (j >= here) break;
          const uint4 xv = x_s[j * pieces + c0 + 32 * u];
          const float2 x0 = unpack(xv.x), x1 = unpack(xv.y), x2 = unpack(xv.z), x3 = unpack(xv.w);
#pragma unroll
          for (int i = 0; i < kRows; ++i) {
            const float2 w0 = unpack(wv[u][i].x), w1 = unpack(wv[u][i].y), w2 = unpack(wv[u][i].z), w3 = unpack(wv[u][i].w);
            float a = acc[i][j];
            a = fmaf(x0.x, w0.x, a);
            a = fmaf(x0.y, w0.y, a);
            a = fmaf(x1.x, w1.x, a);
            a = fmaf(x1.y, w1.y, a);
            a = fmaf(x2.x, w2.x, a);
            a = fmaf(x2.y, w2.y, a);
            a = fmaf(x3.x, w3.x, a);
            acc[i][j] = fmaf(x3.y, w3.y, a);
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < kRows; ++i)
#pragma unroll
      for (int j = 0; j < kTokens; ++j) acc[i][j] = warp_sum(acc[i][j]);
#pragma unroll
    for (int j = 0; j < kTokens; ++j) {
      if (j >= here || lane != j) continue;             // a lane a pair
      const int pair = list_s[first + j];
      if constexpr (kGateUp) {
        const float weight = act.weights ? act.weights[pair] : 1.f;
        const int channel = 16 * blockIdx.x + 2 * warp;           // 2F rows hold F channels, a multiple of 16
        if (row[3] < n)
          *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(out) + (size_t)pair * (n / 2) + channel) =
              __floats2bfloat162_rn(glu(act, acc[0][j], acc[2][j], weight), glu(act, acc[1][j], acc[3][j], weight));
      } else {
        float* dst = reinterpret_cast<float*>(out) + (size_t)pair * n;
#pragma unroll
        for (int i = 0; i < kRows; ++i)
          if (row[i] < n) dst[row[i]] = acc[i][j];
      }
    }
  }
}

}  // namespace cie

using namespace cie;

extern "C" int cie_moe_few_pairs() { return kFewPairs; }

template <bool kGateUp>
static int launch_few(const void* x, const void* w, void* out, const int* ids, int pairs, int top, int experts, int n, int k,
                      const GluAct& act, void* stream) {
  if (pairs <= 0) return 0;
  if (pairs > kFewPairs) CIE_FAIL("moe_few: at most %d pairs, got %d", kFewPairs, pairs);
  if (k % 8 || ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15))
    CIE_FAIL("moe_few: rows of %d elements must be 16-byte aligned", k);
  const size_t smem = (size_t)kTokens * k * sizeof(bf16);
  if (smem > 96 * 1024) CIE_FAIL("moe_few: rows of %d elements do not fit shared memory", k);
  static bool raised = false;
  if (!raised && cudaFuncSetAttribute(moe_few_kernel<kGateUp>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024) != cudaSuccess)
    CIE_FAIL("moe_few: cannot raise the shared memory limit");
  raised = true;
  CIE_LAUNCH("moe_few", moe_few_kernel<kGateUp>, dim3((n + 31) / 32, experts), dim3(kWarps * 32), smem, (cudaStream_t)stream,
             (const bf16*)x, (const bf16*)w, out, ids, pairs, top, n, k, act);
  return 0;
}

// x: [tokens][hidden]; w_gate_up: [experts][2 ff][hidden] interleaved in blocks of 16; act: [tokens * top][ff] by pair; ids:
// [tokens * top].  hidden a multiple of 8, ff a multiple of 16 (clamped, limit, slope, shift, input_weights: GluAct).
extern "C" int cie_moe_gate_up_few(const void* x, const void* w_gate_up, void* act, const int* ids, int tokens, int top,
                                   int experts, int ff, int hidden, int clamped, float limit, float slope, float shift,
                                   const float* input_weights, void* stream) {
  if (ff % 16) CIE_FAIL("moe_gate_up_few: interleaved weights need a multiple of 16 channels, got %d", ff);
  return launch_few<true>(x, w_gate_up, act, ids, tokens * top, top, experts, 2 * ff, hidden,
                          GluAct{clamped, limit, slope, shift, input_weights}, stream);
}

extern "C" int cie_moe_down_few(const void* act, const void* w_down, float* rows, const int* ids, int tokens, int top,
                                int experts, int ff, int hidden, void* stream) {
  return launch_few<false>(act, w_down, rows, ids, tokens * top, top, experts, hidden, ff, GluAct{}, stream);
}

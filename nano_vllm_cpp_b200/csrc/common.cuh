// Shared helpers of the hand-written sm_100a kernels.
//
// Every launcher is an extern "C" function that takes raw device pointers, sizes and a
// cudaStream_t, launches on that stream and returns 0 or a negative NV_ERR_* / positive
// cudaError_t code.  Nothing here allocates device memory: the caller owns every buffer.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <utility>

#define NV_DT_F32 0
#define NV_DT_BF16 1

#define NV_OK 0
#define NV_ERR_BAD_DTYPE (-2)
#define NV_ERR_BAD_SIZE (-3)
#define NV_ERR_UNSUPPORTED (-4)

#define NV_API extern "C" __attribute__((visibility("default")))

#define NV_RETURN_LAST()                          \
  do {                                            \
    cudaError_t e__ = cudaGetLastError();         \
    return e__ == cudaSuccess ? NV_OK : (int)e__; \
  } while (0)

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// Load / store with a run-time dtype code: the plain kernels take it where a template
// parameter would multiply instantiations without making anything faster that matters.
__device__ __forceinline__ float ld_dt(const void* p, int dt, size_t i) {
  return dt == NV_DT_F32 ? ((const float*)p)[i] : __bfloat162float(((const bf16*)p)[i]);
}
__device__ __forceinline__ void st_dt(void* p, int dt, size_t i, float v) {
  if (dt == NV_DT_F32) ((float*)p)[i] = v;
  else ((bf16*)p)[i] = __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// SiLU(g) * u exactly as the reference writes it: g / (1 + expf(-g)) * u  (src/hip_ops.hip:419-429).
__device__ __forceinline__ float silu_mul(float g, float u) { return g / (1.0f + expf(-g)) * u; }

// What a product's launcher takes in its `swiglu` argument: 0 nothing, 1 the SwiGLU pairing of gate and up rows, or a
// unary activation of every output value (after the bias): 2 gelu in its erf form, 3 gelu in its tanh form, 4 silu,
// 5 xIELU with the two positive numbers (p0, p1) that the launcher takes beside it: z > 0: p0 z^2 + z / 2; z <= 0:
// p1 (e^z - 1 - z) + z / 2.
#define NV_EPI_SWIGLU 1
#define NV_EPI_GELU_ERF 2
#define NV_EPI_GELU_TANH 3
#define NV_EPI_SILU 4
#define NV_EPI_XIELU 5
// 6: a second pairing of gate and up rows, with both halves clamped by p0 and the sigmoid's slope p1:
// g = min(g, p0), u = clamp(u, -p0, p0), out = g sigmoid(p1 g) (u + 1).  7: the square of relu.
#define NV_EPI_GLU_CLAMPED 6
#define NV_EPI_RELU2 7
// 8: a third pairing of gate and up rows, gelu in its tanh form on the gate: out = gelu_tanh(g) u.
#define NV_EPI_GEGLU_TANH 8
// 9: silu on the first p0 outputs of a row only; the others pass (a stacked projection of which some columns are activated).
#define NV_EPI_SILU_FIRST 9
#define NV_EPI_LAST NV_EPI_SILU_FIRST
// Which codes pair a gate row with an up row (two accumulators per output), and the pairings themselves.
__host__ __device__ __forceinline__ int epi_pair(int code) {
  return (code == NV_EPI_SWIGLU || code == NV_EPI_GLU_CLAMPED || code == NV_EPI_GEGLU_TANH) ? code : 0;
}
__device__ __forceinline__ float gelu_tanh_of(float z) {
  return 0.5f * z * (1.f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
}
__host__ __device__ __forceinline__ int epi_unary(int code) { return (code >= 2 && !epi_pair(code)) ? code : 0; }
__device__ __forceinline__ float pair_mul(int pair, float g, float u, float p0, float p1) {
  if (pair == NV_EPI_GLU_CLAMPED) {
    g = fminf(g, p0);
    u = fminf(fmaxf(u, -p0), p0);
    return g / (1.0f + expf(-p1 * g)) * (u + 1.0f);
  }
  if (pair == NV_EPI_GEGLU_TANH) return gelu_tanh_of(g) * u;
  return silu_mul(g, u);
}
__device__ __forceinline__ float epilogue_act(int act, float v, float p0 = 0.f, float p1 = 0.f) {
  if (act == 0) return v;
  if (act == NV_EPI_RELU2) { v = fmaxf(v, 0.f); return v * v; }
  if (act == NV_EPI_XIELU) return v > 0.f ? fmaf(p0 * v, v, 0.5f * v) : fmaf(p1, expm1f(v) - v, 0.5f * v);
  if (act == NV_EPI_GELU_ERF) return 0.5f * v * (1.f + erff(v * 0.70710678118654752440f));
  if (act == NV_EPI_GELU_TANH) return gelu_tanh_of(v);
  return v / (1.f + expf(-v));
}

// The unary activation of output feature n, for the codes that do not treat all features alike.
__device__ __forceinline__ int epi_at(int act, int n, float p0) {
  return act == NV_EPI_SILU_FIRST ? (n < (int)p0 ? NV_EPI_SILU : 0) : act;
}

// What multiplies a query head's attention output before it is stored: sigmoid of `gate[t * ld + h]` (t the batch row, h
// the query head), or one without a gate (gate == nullptr).
struct HeadGate {
  const float* gate;
  long long ld;
};
__device__ __forceinline__ float head_gate_of(const HeadGate& g, long long t, int h) {
  return g.gate ? 1.f / (1.f + expf(-g.gate[t * g.ld + h])) : 1.f;
}

// What the distance between a row and a key gives to their score, after the cap and before the softmax: -slope[h] * n, and
// entry min(n, last) of the head's row of a table, for query head h and distance n (either array may be nullptr).  A table's
// row has NV_BIAS_PAD further entries on both sides (copies of its ends), so that a run of neighbouring keys around either end
// can be read without clamping every index.
#define NV_BIAS_PAD 64
struct ScoreBias {
  const float* slope;
  const float* table;
  int last;
};
__device__ __forceinline__ const float* bias_row(const ScoreBias& b, int h) {      // the row's entry 0
  return b.table ? b.table + (size_t)h * (b.last + 1 + 2 * NV_BIAS_PAD) + NV_BIAS_PAD : nullptr;
}
__device__ __forceinline__ float score_bias_of(const ScoreBias& b, int h, int n) {
  float v = b.slope ? -b.slope[h] * (float)n : 0.f;
  if (b.table) v += bias_row(b, h)[min(n, b.last)];
  return v;
}
// The first position that a row at position p sees: a sliding window (0: none), or the start of its chunk (0: no chunks).
__host__ __device__ __forceinline__ int first_visible(int p, int window, int chunk) {
  if (chunk > 0) return p / chunk * chunk;
  return window > 0 && p + 1 > window ? p + 1 - window : 0;
}
__device__ __forceinline__ float ex2_fast(float x) {         // 2^x by the special-function unit
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// A score on its way to base-2 units in the tensor-core kernels.  cap tanh(x / cap) = cap - 2 cap / (e^(2 x / cap) + 1), whose
// absolute error is a few units of the cap's last place, as the difference's is whatever x is.
struct ScoreMap {
  float in;                 // without a cap: scale * log2(e)
  float cap_k, cap1, cap2;  // with a cap (cap1 > 0): 2 log2(e) scale / cap, cap log2(e), 2 cap log2(e)
};
static inline ScoreMap score_map(float scale, float softcap) {
  const float l2e = 1.4426950408889634f;
  ScoreMap m = {scale * l2e, 0.f, 0.f, 0.f};
  if (softcap > 0.f) {
    m.cap_k = 2.f * l2e * scale / softcap;
    m.cap1 = softcap * l2e;
    m.cap2 = 2.f * softcap * l2e;
  }
  return m;
}
__device__ __forceinline__ float capped_log2(const ScoreMap& m, float s) {
  return fmaf(-m.cap2, rcp_fast(ex2_fast(s * m.cap_k) + 1.f), m.cap1);
}

// Programmatic dependent launch.  A kernel launched with the programmatic-serialization attribute may start
// while the kernel before it in the stream still runs; what it reads of that kernel's results, and whatever it
// writes, must come after grid_dep_wait(), which returns once the earlier kernel has finished and its writes
// are visible.  grid_dep_launch() in the earlier kernel says "my dependents may be scheduled now" (once every
// CTA has said so or exited); without it they are scheduled as its CTAs exit.  Both are no-ops for kernels
// launched the ordinary way.
__device__ __forceinline__ void grid_dep_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void grid_dep_launch() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

// Launches `kernel` as a programmatic dependent of the kernel before it on the stream (an ordinary launch
// when nv_set_dependent_launch(0) was called).  Such a kernel must call grid_dep_wait() before it reads anything
// an earlier kernel of the step wrote and before it writes anything, and calls grid_dep_launch() right after,
// so that at most one kernel is ever set up ahead of the one that runs: everything older has finished by then.
// Grids of more than NV_DEP_MAX_BLOCKS blocks are launched the ordinary way: their waiting blocks would crowd
// the multiprocessors on which the kernel before them is still finishing (measured: a prompt of 2,048 tokens
// ran 7 % slower with every kernel a dependent), and a launch latency is nothing beside such a kernel's time.
constexpr unsigned NV_DEP_MAX_BLOCKS = 2048;
extern int g_nv_dependent_launch;
template <typename... Exp, typename... Act>
static inline cudaError_t launch_dep(void (*kernel)(Exp...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                     Act&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  const unsigned long long blocks = (unsigned long long)grid.x * grid.y * grid.z;
  attr[0].val.programmaticStreamSerializationAllowed = (g_nv_dependent_launch && blocks <= NV_DEP_MAX_BLOCKS) ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<Exp>(args)...);
}
#define NV_RETURN_IF(e)                            \
  do {                                             \
    cudaError_t e2__ = (e);                        \
    if (e2__ != cudaSuccess) return (int)e2__;     \
  } while (0)

static inline int dt_ok(int dt) { return dt == NV_DT_F32 || dt == NV_DT_BF16; }

// Shared helpers of the sm_100a kernels: element types, warp reductions, error reporting.
//
// Every entry point is `extern "C"`, takes raw device pointers, sizes and a stream, launches
// asynchronously on that stream and returns 0, or returns non-zero after recording a message
// that leb_last_error() hands out.  Nothing here allocates device memory.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#define LEB_API extern "C" __attribute__((visibility("default")))

// element type codes shared with the Python side
enum LebDtype { LEB_F32 = 0, LEB_BF16 = 1 };

int leb_fail(const char* fmt, ...);  // records the message, returns 1

// Kernels launched by this library since it was loaded (each check stands for one launch).
extern long long g_leb_launches;

#define LEB_CHECK_LAUNCH(name)                                                        \
  do {                                                                                \
    cudaError_t e_ = cudaGetLastError();                                              \
    if (e_ != cudaSuccess) return leb_fail("%s: %s", name, cudaGetErrorString(e_));   \
    g_leb_launches++;                                                                 \
  } while (0)

// Launch with programmatic dependent launch: the kernel may be scheduled while the one before
// it on the stream is still running, so its start-up (and whatever it does before pdl_wait())
// overlaps the tail of its predecessor.  A decode step is a chain of ~100 short kernels; this
// takes the launch gap out of every link.  Kernels launched this way call pdl_wait() before they
// touch anything the previous kernel wrote, and write nothing before it.
extern int g_leb_pdl;   // 1: use the attribute (default), 0: plain launches
template <typename... KArgs, typename... Args>
static inline cudaError_t leb_launch(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                     cudaStream_t st, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = g_leb_pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kern, static_cast<KArgs>(args)...);
}
// Launches of a scope without programmatic dependent launch (strictly after their predecessor).
struct LebPlainLaunches {
  int saved;
  bool off;
  explicit LebPlainLaunches(bool turn_off) : saved(g_leb_pdl), off(turn_off) { if (off) g_leb_pdl = 0; }
  ~LebPlainLaunches() { if (off) g_leb_pdl = saved; }
};
// silu(g) * u.  The bfloat16 products' epilogues take 2^x and the reciprocal from the special
// function unit (relative error about 1e-6, far below the rounding of the bfloat16 they store):
// with exact expf and division an epilogue of a few warps is bound by its instructions.
template <typename T>
__device__ __forceinline__ float silu_mul(float g, float u) {
  if (sizeof(T) == 2) return __fdividef(g, 1.0f + __expf(-g)) * u;
  return g / (1.0f + expf(-g)) * u;
}
// A gated epilogue (code 2: act(gate) * up over interleaved weight rows) names its activation in the
// upper bits of the epilogue code the kernels get: 0 silu, 1 the tanh form of gelu, 2 the clamped
// sigmoid form g' sigmoid(1.702 g') (u' + 1) with g' = min(g, L), u' = clamp(u, -L, L), whose limit L
// rides above the code as the upper 16 bits of its float (a limit that bfloat16 holds exactly).  The
// entry points take the same combined code, check it, and hand it on through LEB_EPI_ARG at the launch.
extern thread_local int g_leb_gate_act;
#define LEB_EPI_ARG(e) ((e) | (g_leb_gate_act << 8))
#define LEB_GATE_ACT_OK(act, epi) ((act) == 0 || (((act) == 1 || ((act) & 255) == 2) && (epi) == 2))
template <typename T>
__device__ __forceinline__ float gate_mul(float g, float u, int act) {
  if ((act & 255) == 2) {
    const float lim = __uint_as_float(((unsigned)act >> 8) << 16);
    g = fminf(g, lim);
    u = fminf(fmaxf(u, -lim), lim);
    if (sizeof(T) == 2) return __fdividef(g, 1.0f + __expf(-1.702f * g)) * (u + 1.0f);
    return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
  }
  if (act == 1) {
    const float z = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    float t;
    if (sizeof(T) == 2) asm("tanh.approx.f32 %0, %1;" : "=f"(t) : "f"(z));   // as silu_mul: far below bfloat16 rounding
    else t = tanhf(z);
    return 0.5f * g * (1.0f + t) * u;
  }
  return silu_mul<T>(g, u);
}
// An activation without a gate in a storing epilogue (code 0) of the bfloat16 products that take it (the weight
// stream of a decode step and the tcgen05 products, dense and grouped): code LEB_PLAIN_ACT_BASE + a in the place of the gated activation, a as
// leb_activation counts them (0 the erf form of gelu, 1 the square of relu, 2 the tanh form of gelu, 3 silu).  The
// exact functions, as the activation kernel uses them: a row gives the same numbers through either.
#define LEB_PLAIN_ACT_BASE 16
#define LEB_PLAIN_ACT_OK(act, epi) ((act) >= LEB_PLAIN_ACT_BASE && (act) < LEB_PLAIN_ACT_BASE + 4 && (epi) == 0)
__device__ __forceinline__ float plain_act(float z, int act) {
  const int a = act - LEB_PLAIN_ACT_BASE;
  if (a == 0) return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f));
  if (a == 1) { const float t = fmaxf(z, 0.f); return t * t; }
  if (a == 2) return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
  return z / (1.0f + expf(-z));
}
// Device side.  pdl_trigger(): the next kernel on the stream may be scheduled (once every block
// of this one has said so); it then runs its own start-up and waits in its pdl_wait() until this
// kernel has completed.  Said first thing, even before this kernel's own wait: a product two
// launches down the stream can then fetch its weights while the one before it still runs (its
// wait covers everything before it, since the kernel it waits for has itself waited).
// pdl_wait(): wait until the previous kernel has completed and its writes are visible (a no-op
// for a plain launch).
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() {
  pdl_trigger();
  asm volatile("griddepcontrol.wait;" ::: "memory");
}

#define LEB_REQUIRE(cond, ...)                 \
  do {                                         \
    if (!(cond)) return leb_fail(__VA_ARGS__); \
  } while (0)

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// Four neighbouring numbers as floats (16 bytes of float, 8 of bfloat16; aligned to that).
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 c = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, c.x, c.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
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

// Sum over a block of up to 1024 threads; every thread gets the result.  `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();  // `red` may still be read from an earlier call
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nw ? red[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

// First key position the query at `pos` reads: 0, the start of its window of `window` positions, or the start of its
// chunk of `chunk` positions counted from the sequence's first (each where positive; never falls as pos grows).
__device__ __forceinline__ int first_key(int pos, int window, int chunk) {
  int lo = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
  if (chunk > 0) lo = max(lo, pos - pos % chunk);
  return lo;
}

// The factor sigmoid(gate) of a head's result: one per (row, head), or with `elem` one per dimension of the head
// (gate [rows, heads, width]).
template <typename T>
__device__ __forceinline__ float head_gate(const T* gate, size_t row, int stride, int h, int d, int width, int elem) {
  const float z = to_f32(gate[row * stride + (elem ? h * width + d : h)]);
  return 1.0f / (1.0f + expf(-z));
}

// The factor on a query at position p: 1 + coef ln(floor((p + 1) / every) + 1).
__device__ __forceinline__ float query_temperature(int p, float coef, float every) {
  return coef != 0.f ? 1.0f + coef * logf(floorf((float)(p + 1) / every) + 1.0f) : 1.0f;
}

// A softmax row summed as (m, l) = (reference maximum, sum of e^(s - m)) takes one more logit `sink` into its denominator
// (a logit without a key or a value): returns what the row's weighted sum of values is multiplied by.
__device__ __forceinline__ float sink_quotient(float m, float l, float sink) {
  const float top = fmaxf(m, sink), f = expf(m - top);
  return f / (l * f + expf(sink - top));
}

static inline int ceil_div(int a, int b) { return (a + b - 1) / b; }

// SMs of the current device, asked once per device (device_info.cu); launch shapes that are
// chosen for "a wave of blocks" use it.
extern "C" int leb_sm_count();
static inline int sm_count() {
  int n = leb_sm_count();
  return n > 0 ? n : 1;
}

// Shared helpers of the sm_100a kernels: storage-type load/store (activations, weights
// and caches are float or bfloat16; all arithmetic is float), warp/block reductions and
// the C-ABI launch convention.  Every exported launcher returns a cudaError_t as int
// (0 = launched) and never synchronises or allocates.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define PMM_DTYPE_F32 0
#define PMM_DTYPE_BF16 1
#define PMM_ERR_BAD_ARGUMENT 1001  // outside the cudaError_t range that launches return

#define PMM_EXPORT extern "C" __attribute__((visibility("default")))

namespace pmm {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Two and four neighbouring elements (the pointer on a boundary of as many).
__device__ __forceinline__ float2 ldf2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ldf2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void stf2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void stf2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }
__device__ __forceinline__ float4 ldf4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ldf4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void stf4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void stf4(__nv_bfloat16* p, float4 v) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = raw;
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

// Sum over the block; `red` is shared memory for 32 floats.  Every thread gets the total.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarp = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();  // protects `red` against a previous use
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = (lane < nwarp) ? red[lane] : 0.f;
  t = warp_sum(t);
  return t;
}

// Two sums over the block at once; `red` is shared memory for 64 floats.
__device__ __forceinline__ float2 block_sum2(float2 v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarp = (blockDim.x + 31) >> 5;
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  __syncthreads();  // protects `red` against a previous use
  if (lane == 0) {
    red[warp] = v.x;
    red[32 + warp] = v.y;
  }
  __syncthreads();
  return make_float2(warp_sum(lane < nwarp ? red[lane] : 0.f), warp_sum(lane < nwarp ? red[32 + lane] : 0.f));
}

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// For results that are stored as bfloat16: relative error about 1e-6, three instructions' worth
// of special-function work instead of a full-precision exponential and division.
__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.f + __expf(-x)); }

// The exact (erf) form of GELU: z/2 (1 + erf(z / sqrt 2)).
__device__ __forceinline__ float gelu_erf_f(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }
// For results that are stored as bfloat16: with x = |z| / sqrt 2 and t = 1 / (1 + 0.3275911 x),
// erfc(x) = (a1 t + ... + a5 t^5) e^(-x^2) to 1.5e-7 (Abramowitz and Stegun, Handbook of Mathematical Functions, 7.1.26).
__device__ __forceinline__ float gelu_erf_fast(float z) {
  const float x = fabsf(z) * 0.70710678118654752f;
  const float t = __fdividef(1.f, 1.f + 0.3275911f * x);
  const float poly = t * (0.254829592f + t * (-0.284496736f + t * (1.421413741f + t * (-1.453152027f + t * 1.061405429f))));
  const float half = 0.5f * z * poly * __expf(-x * x);  // z/2 erfc(x)
  return z >= 0.f ? z - half : half;
}

// v if v>20; exp(v) if v<-20; log1p(exp(v)) otherwise.
__device__ __forceinline__ float softplus_f(float v) {
  if (v > 20.f) return v;
  if (v < -20.f) return expf(v);
  return log1pf(expf(v));
}

// The first key that the token at `pos` may see: window > 0 the last `window` keys, window < 0 the keys of its own
// chunk of -window positions (counted from position 0), window == 0 every key.  Does not fall as pos grows.
__device__ __forceinline__ int first_visible(int pos, int window) {
  if (window > 0) return max(0, pos - window + 1);
  return window < 0 ? pos - pos % -window : 0;
}

// Softplus and exponential of the recurrences' walks, in the type the walk computes in (float, or double for the
// float storage type).
template <typename ACC>
__device__ __forceinline__ ACC scan_softplus(ACC v);
template <>
__device__ __forceinline__ float scan_softplus<float>(float v) { return softplus_f(v); }
template <>
__device__ __forceinline__ double scan_softplus<double>(double v) {
  if (v > 40.0) return v;
  return log1p(exp(v));
}
__device__ __forceinline__ float scan_exp(float v) { return expf(v); }
__device__ __forceinline__ double scan_exp(double v) { return exp(v); }

inline int launch_status() { return static_cast<int>(cudaGetLastError()); }

// Programmatic dependent launch.  A kernel started with launch_pdl may begin while the kernel
// before it on the stream is still running; pdl_wait() inside it returns once that kernel has
// finished and its writes are visible, so everything a kernel does before pdl_wait() must not
// touch memory that other kernels write (reading constant weights is fine).
// pdl_launch_dependents() lets the next kernel of the stream start its own preamble early.
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

template <typename... KArgs, typename... Args>
inline void launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                       Args&&... args) {
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr{};
  attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr.val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = &attr;
  cfg.numAttrs = 1;
  cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);  // errors surface in launch_status()
}

}  // namespace pmm

// Calls FN<float>(...) or FN<__nv_bfloat16>(...) by dtype code.
#define PMM_DISPATCH_DTYPE(code, S, ...)          \
  do {                                            \
    if ((code) == PMM_DTYPE_F32) {                \
      using S = float;                            \
      __VA_ARGS__;                                \
    } else if ((code) == PMM_DTYPE_BF16) {        \
      using S = __nv_bfloat16;                    \
      __VA_ARGS__;                                \
    } else {                                      \
      return PMM_ERR_BAD_ARGUMENT;                \
    }                                             \
  } while (0)

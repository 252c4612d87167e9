// seq_common.cuh — helpers shared by the ragged-batch kernels of the hybrid layer stacks (seq_mixers.cu,
// parallel_mixers.cu): dispatch over the activation type, gate functions in 32-bit, vector loads and stores as fp32.
#pragma once
#include "sxb_common.cuh"

#define SEQMIX_DISPATCH(dtype, ...)                \
  do {                                             \
    if ((dtype) == 0) {                         \
      using T = float;                             \
      __VA_ARGS__;                                 \
    } else if ((dtype) == 2) {                 \
      using T = __nv_bfloat16;                     \
      __VA_ARGS__;                                 \
    } else {                                       \
      return SXB_ERR_UNSUPPORTED;                  \
    }                                              \
  } while (0)

namespace sxb {
namespace seqmix {

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 30.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

template <typename T>
__device__ __forceinline__ float4 load4_f32(const T* p);
template <>
__device__ __forceinline__ float4 load4_f32<float>(const float* p) {
  return *reinterpret_cast<const float4*>(p);
}
template <>
__device__ __forceinline__ float4 load4_f32<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x);
  const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}

template <typename T>
__device__ __forceinline__ void load8_f32(const T* p, float* o);
template <>
__device__ __forceinline__ void load8_f32<float>(const float* p, float* o) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  o[0] = a.x, o[1] = a.y, o[2] = a.z, o[3] = a.w, o[4] = b.x, o[5] = b.y, o[6] = b.z, o[7] = b.w;
}
template <>
__device__ __forceinline__ void load8_f32<__nv_bfloat16>(const __nv_bfloat16* p, float* o) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) o[2 * i] = __low2float(h[i]), o[2 * i + 1] = __high2float(h[i]);
}

template <typename T>
__device__ __forceinline__ void store4_f32(T* p, float4 v);
template <>
__device__ __forceinline__ void store4_f32<float>(float* p, float4 v) {
  *reinterpret_cast<float4*>(p) = v;
}
template <>
__device__ __forceinline__ void store4_f32<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

template <typename T>
__device__ __forceinline__ void store8_f32(T* p, const float* o);
template <>
__device__ __forceinline__ void store8_f32<float>(float* p, const float* o) {
  reinterpret_cast<float4*>(p)[0] = make_float4(o[0], o[1], o[2], o[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(o[4], o[5], o[6], o[7]);
}
template <>
__device__ __forceinline__ void store8_f32<__nv_bfloat16>(__nv_bfloat16* p, const float* o) {
  *reinterpret_cast<uint4*>(p) =
      make_uint4(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]), pack_bf16(o[4], o[5]), pack_bf16(o[6], o[7]));
}

// Sums of two numbers over the block, both at once (blockDim.x <= 1024 and a multiple of 32).
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* smem /* >= 32 */) {
  a = warp_sum(a), b = warp_sum(b);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();
  if (l == 0) smem[w] = make_float2(a, b);
  __syncthreads();
  const int nw = (blockDim.x + 31) >> 5;
  const float2 r = (l < nw) ? smem[l] : make_float2(0.f, 0.f);
  return make_float2(warp_sum(r.x), warp_sum(r.y));
}

}  // namespace seqmix
}  // namespace sxb

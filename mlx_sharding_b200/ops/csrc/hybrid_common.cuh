// Device helpers shared by the hybrid-stack kernel files (hybrid.cu, diffattn.cu): typed loads / stores of activations (bf16 or float),
// warp and block reductions, the row -> sequence search of a ragged step, and the activation-type dispatch of the launchers.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

namespace b200 {
namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
// activations round to AT between a projection and its nonlinearity, as an unfused graph does
template <typename T> __device__ __forceinline__ float rnd(float v);
template <> __device__ __forceinline__ float rnd<float>(float v) { return v; }
template <> __device__ __forceinline__ float rnd<__nv_bfloat16>(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }

// 16 bytes of activations -> floats
template <typename T> __device__ __forceinline__ void unpack16(const uint4& v, float* dst);
template <> __device__ __forceinline__ void unpack16<float>(const uint4& v, float* dst) {
  dst[0] = __uint_as_float(v.x); dst[1] = __uint_as_float(v.y); dst[2] = __uint_as_float(v.z); dst[3] = __uint_as_float(v.w);
}
template <> __device__ __forceinline__ void unpack16<__nv_bfloat16>(const uint4& v, float* dst) {
  const unsigned w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { dst[2 * i] = __uint_as_float(w[i] << 16); dst[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
}

// four adjacent activations <-> floats (pointers aligned to four entries)
template <typename T> __device__ __forceinline__ void load4(const T* p, float* f);
template <> __device__ __forceinline__ void load4<float>(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
template <> __device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float* f) {
  const uint2 a = *reinterpret_cast<const uint2*>(p);
  f[0] = __uint_as_float(a.x << 16); f[1] = __uint_as_float(a.x & 0xffff0000u); f[2] = __uint_as_float(a.y << 16); f[3] = __uint_as_float(a.y & 0xffff0000u);
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float* f);
template <> __device__ __forceinline__ void store4<float>(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float* f) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(f[0], f[1]), hi = __floats2bfloat162_rn(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(reinterpret_cast<unsigned&>(lo), reinterpret_cast<unsigned&>(hi));
}

// two floats in one 64-bit register: packed multiply and multiply-add
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(reinterpret_cast<unsigned long long&>(r)) : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)));
  return r;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(reinterpret_cast<unsigned long long&>(r))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)), "l"(reinterpret_cast<unsigned long long&>(c)));
  return r;
}

__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return v > 30.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
__device__ __forceinline__ float gelu_erf_f(float z) { return 0.5f * z * (1.f + erff(z * 0.7071067811865476f)); }

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
// Sums of NV values over LK lanes, every lane gets all of them: each level sends half of the values that are left one way and keeps the other
// half (NV - 1 shuffles in all instead of NV log2 LK), then the totals are handed round.
template <int NV, int LK> __device__ __forceinline__ void sum_over_lanes(float (&v)[NV], int lane) {
  int left = NV;
#pragma unroll
  for (int w = 1; w < LK; w <<= 1) {
    if (left > 1) {
      left >>= 1;
      const bool up = lane & w;
#pragma unroll
      for (int i = 0; i < NV / 2; ++i)
        if (i < left) {
          const float send = up ? v[i] : v[i + left], keep = up ? v[i + left] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, w);
        }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], w);
    }
  }
  float r[NV];
#pragma unroll
  for (int x = 0; x < NV; ++x) {
    int src = 0, n = NV;
#pragma unroll
    for (int w = 1; w < LK; w <<= 1)
      if (n > 1) { n >>= 1; if (x & n) src |= w; }
    r[x] = __shfl_sync(0xffffffffu, v[x % left], src, LK);
  }
#pragma unroll
  for (int x = 0; x < NV; ++x) v[x] = r[x];
}
// sum over the block (blockDim.x <= 1024, multiple of 32); every thread gets the result
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < nw ? red[l] : 0.f;
  return warp_sum(t);
}
// sequence of row t: largest b with cu[b] <= t
__device__ __forceinline__ int seq_of(const int* cu, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

inline cudaError_t last() { return cudaGetLastError(); }
#define AT_DISPATCH(f32, ...)                                      \
  do {                                                             \
    if (f32) { using AT = float; __VA_ARGS__; }                    \
    else { using AT = __nv_bfloat16; __VA_ARGS__; }                \
  } while (0)


}  // namespace
}  // namespace b200

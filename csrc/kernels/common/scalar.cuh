// Element access and block reductions shared by the kernels that run on bf16 or fp32 activations: arithmetic is always
// fp32, the element type only says how activations are stored.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace lt {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// The value as the element type holds it (what a store followed by a load gives).
__device__ __forceinline__ float round_as(const float*, float v) { return v; }
__device__ __forceinline__ float round_as(const __nv_bfloat16*, float v) { return __bfloat162float(__float2bfloat16(v)); }

// Four neighbouring elements; p is aligned to four elements.
__device__ __forceinline__ float4 ldf4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ldf4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void stf4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void stf4(__nv_bfloat16* p, float4 v) {
  uint2 u;
  *reinterpret_cast<__nv_bfloat162*>(&u.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&u.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = u;
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

// Sums of N (a power of two up to 32) values over the warp with N - 1 + log2(32 / N) exchanges instead of 5 N: lane l gets
// the sum of value l % N.  v is used up.
template <int N>
__device__ __forceinline__ float warp_sum_each(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int half = N / 2; half >= 1; half >>= 1) {
    const bool up = (lane & half) != 0;
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float keep = up ? v[i + half] : v[i], give = up ? v[i] : v[i + half];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, half);
    }
  }
  float r = v[0];
#pragma unroll
  for (int o = N; o < 32; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
  return r;
}

// Eight neighbouring elements as fp32; p is aligned to eight elements.
__device__ __forceinline__ void ldf8(const float* p, float (&v)[8]) {
  const float4 a = ldf4(p), b = ldf4(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void ldf8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x;
    v[2 * i + 1] = f.y;
  }
}

// Sums of two values over the block, returned to every thread; red holds 64 floats and is free again on return.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  if (lane == 0) { red[warp] = a; red[32 + warp] = b; }
  __syncthreads();
  float sa = 0.f, sb = 0.f;
  for (int w = 0; w < nw; ++w) { sa += red[w]; sb += red[32 + w]; }
  __syncthreads();
  return make_float2(sa, sb);
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// SiLU for results that leave as bf16: the quick exponential and quotient (a few units in the last place of fp32).
__device__ __forceinline__ float silu_quick_f(float x) { return __fdividef(x, 1.f + __expf(-x)); }
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

}  // namespace lt

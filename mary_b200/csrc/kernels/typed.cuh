// Scalar access helpers for kernels that are instantiated for bf16 and for 32-bit storage.
#pragma once
#include "common.cuh"

namespace mary {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// 16 bytes of storage as floats: 8 bf16 or 4 f32 values.
template <typename T> struct Pack;
template <> struct Pack<float> { static constexpr int N = 4; };
template <> struct Pack<__nv_bfloat16> { static constexpr int N = 8; };
__device__ __forceinline__ void unpack16(const uint4& v, float (&f)[4]) {
  f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
}
__device__ __forceinline__ void unpack16(const uint4& v, float (&f)[8]) {
  const __nv_bfloat162* h = (const __nv_bfloat162*)&v;
#pragma unroll
  for (int j = 0; j < 4; ++j) { const float2 t = __bfloat1622float2(h[j]); f[2 * j] = t.x; f[2 * j + 1] = t.y; }
}
__device__ __forceinline__ uint4 pack16(const float (&f)[4]) {
  return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
}
__device__ __forceinline__ uint4 pack16(const float (&f)[8]) {
  uint4 v;
  __nv_bfloat162* h = (__nv_bfloat162*)&v;
#pragma unroll
  for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(f[2 * j], f[2 * j + 1]);
  return v;
}

// E consecutive values (E = 4: one 8- or 16-byte access, aligned) as floats.
template <typename T, int E> __device__ __forceinline__ void load_e(const T* p, float (&f)[E]) {
  if constexpr (E == 4 && sizeof(T) == 2) {
    const uint2 v = *(const uint2*)p;
    const __nv_bfloat162* h = (const __nv_bfloat162*)&v;
    const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else if constexpr (E == 4) {
    const float4 v = *(const float4*)p;
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
#pragma unroll
    for (int j = 0; j < E; ++j) f[j] = to_f<T>(p[j]);
  }
}
template <typename T, int E> __device__ __forceinline__ void store_e(T* p, const float (&f)[E]) {
  if constexpr (E == 4 && sizeof(T) == 2) {
    uint2 v;
    __nv_bfloat162* h = (__nv_bfloat162*)&v;
    h[0] = __floats2bfloat162_rn(f[0], f[1]); h[1] = __floats2bfloat162_rn(f[2], f[3]);
    *(uint2*)p = v;
  } else if constexpr (E == 4) {
    *(float4*)p = make_float4(f[0], f[1], f[2], f[3]);
  } else {
#pragma unroll
    for (int j = 0; j < E; ++j) p[j] = from_f<T>(f[j]);
  }
}

// E values, one 16-byte access of bf16 or two of f32 when E = 8, see load_e otherwise.
template <typename T, int E> __device__ __forceinline__ void load_v(const T* p, float (&f)[E]) {
  if constexpr (E == 8 && sizeof(T) == 2) unpack16(*(const uint4*)p, f);
  else if constexpr (E == 8) {
    *(float4*)f = *(const float4*)p;
    *(float4*)(f + 4) = *(const float4*)(p + 4);
  } else {
    load_e<T, E>(p, f);
  }
}
template <typename T, int E> __device__ __forceinline__ void store_v(T* p, const float (&f)[E]) {
  if constexpr (E == 8 && sizeof(T) == 2) *(uint4*)p = pack16(f);
  else if constexpr (E == 8) {
    *(float4*)p = *(const float4*)f;
    *(float4*)(p + 4) = *(const float4*)(f + 4);
  } else {
    store_e<T, E>(p, f);
  }
}

// Exact forms (these files are compiled without fast math): logistic function, SiLU, softplus and the log of the logistic function.
__device__ __forceinline__ float sigmoid_x(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_x(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_x(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_sigmoid_x(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

// The same by storage type: exact for 32-bit models, the hardware's fast exponential / logarithm / divide (a few units in the last place
// of a 32-bit result) for bf16 models.
template <typename T> __device__ __forceinline__ float exp_t(float x) {
  if constexpr (sizeof(T) == 4) return expf(x);
  else return __expf(x);
}
template <typename T> __device__ __forceinline__ float silu_t(float x) {
  if constexpr (sizeof(T) == 4) return silu_x(x);
  else return __fdividef(x, 1.0f + __expf(-x));
}
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (sizeof(T) == 4) return sigmoid_x(x);
  else return __fdividef(1.0f, 1.0f + __expf(-x));
}
template <typename T> __device__ __forceinline__ float log_sigmoid_t(float x) {
  if constexpr (sizeof(T) == 4) return log_sigmoid_x(x);
  else return fminf(x, 0.f) - __logf(1.0f + __expf(-fabsf(x)));
}

// One halving step of a reduction over lanes: of N values a lane keeps the half its lane bit selects and adds what its partner sends.
template <int N>
__device__ __forceinline__ void halve(float* v, int lane, int bit) {
  const bool up = (lane & bit) != 0;
#pragma unroll
  for (int i = 0; i < N / 2; ++i) {
    const float send = up ? v[i] : v[i + N / 2], keep = up ? v[i + N / 2] : v[i];
    v[i] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
  }
}

__device__ __forceinline__ float block_sum_x(float v, float* red) {      // red: 32 floats of shared memory
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = (l < (int)(blockDim.x >> 5)) ? red[l] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

}  // namespace mary

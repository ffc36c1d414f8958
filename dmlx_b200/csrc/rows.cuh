// Device helpers of the kernels that stand between a decoder's matmuls: rows of a matmul's result wherever they are, vectors
// of 1 or 4 elements of either number format, warp and block sums.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

// Result of a matmul, row by row: f32 split-K partial tiles (ws) or rows the matmul wrote itself (y).
struct MatSrc {
  const float* ws = nullptr;
  int splits = 0, tn = 0, tts = 0;
  const void* y = nullptr;
  int y_stride = 0;
};

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <int VEC>
struct Vec { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ Vec<VEC> load_vec(const float* p) {
  Vec<VEC> r;
  if constexpr (VEC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ Vec<VEC> load_vec(const __nv_bfloat16* p) {
  Vec<VEC> r;
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    r.v[0] = __uint_as_float(u.x << 16); r.v[1] = __uint_as_float(u.x & 0xFFFF0000u);
    r.v[2] = __uint_as_float(u.y << 16); r.v[3] = __uint_as_float(u.y & 0xFFFF0000u);
  } else {
    r.v[0] = __bfloat162float(*p);
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* p, const Vec<VEC>& x) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
  else *p = x.v[0];
}
template <int VEC>
__device__ __forceinline__ void store_vec(__nv_bfloat16* p, const Vec<VEC>& x) {
  if constexpr (VEC == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(x.v[0], x.v[1]), b = __floats2bfloat162_rn(x.v[2], x.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16(x.v[0]);
  }
}

// A vector as it lies in memory, for loads that are to be in flight while something else happens.
template <typename T, int VEC>
struct Raw;
template <>
struct Raw<float, 4> { float4 r; };
template <>
struct Raw<float, 1> { float r; };
template <>
struct Raw<__nv_bfloat16, 4> { uint2 r; };
template <>
struct Raw<__nv_bfloat16, 1> { __nv_bfloat16 r; };
template <typename T, int VEC>
__device__ __forceinline__ Raw<T, VEC> load_raw(const T* p) { return *reinterpret_cast<const Raw<T, VEC>*>(p); }
template <typename T, int VEC>
__device__ __forceinline__ Vec<VEC> widen(const Raw<T, VEC>& raw) { return load_vec<VEC>(reinterpret_cast<const T*>(&raw)); }

// Columns c .. c + VEC - 1 of one row; the splits are summed in split order.
template <typename T, int VEC>
__device__ __forceinline__ Vec<VEC> mat_value(const MatSrc& s, int row, int c) {
  if (!s.ws) return load_vec<VEC>((const T*)s.y + (size_t)row * s.y_stride + c);
  const int nt = c >> 7, r = c & 127, tt = row / s.tn, tr = row - tt * s.tn;
  const float* p = s.ws + (((size_t)(nt * s.tts + tt) * s.splits) * s.tn + tr) * 128 + r;
  Vec<VEC> acc = load_vec<VEC>(p);
  for (int i = 1; i < s.splits; ++i) {
    const Vec<VEC> b = load_vec<VEC>(p + (size_t)i * s.tn * 128);
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc.v[e] += b.v[e];
  }
  return acc;
}

// The same with the loads of up to AHEAD splits in flight, for kernels of few rows.
template <typename T, int VEC, int AHEAD>
__device__ __forceinline__ Vec<VEC> mat_value_ahead(const MatSrc& s, int row, int c) {
  if (!s.ws) return load_vec<VEC>((const T*)s.y + (size_t)row * s.y_stride + c);
  const int nt = c >> 7, r = c & 127, tt = row / s.tn, tr = row - tt * s.tn;
  const float* p = s.ws + (((size_t)(nt * s.tts + tt) * s.splits) * s.tn + tr) * 128 + r;
  Vec<VEC> acc{};
  for (int i = 0; i < s.splits; i += AHEAD) {
    Vec<VEC> b[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      b[u] = Vec<VEC>{};
      if (i + u < s.splits) b[u] = load_vec<VEC>(p + (size_t)(i + u) * s.tn * 128);
    }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc.v[e] += b[u].v[e];
    }
  }
  return acc;
}

// Sigmoid for results that are kept as T: bf16 ones take the hardware's exponential and reciprocal.
template <typename T>
__device__ __forceinline__ float sigmoid_for(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.0f, 1.0f + __expf(-z));
  else return 1.0f / (1.0f + expf(-z));
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Four sums at once; part holds a number of the block's warps.
__device__ __forceinline__ float4 block_sum4(float4 v, float4* part) {
  v = make_float4(warp_sum(v.x), warp_sum(v.y), warp_sum(v.z), warp_sum(v.w));
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  const int lane = threadIdx.x & 31;
  v = lane < (int)(blockDim.x >> 5) ? part[lane] : make_float4(0.f, 0.f, 0.f, 0.f);  // (every warp for itself)
  return make_float4(warp_sum(v.x), warp_sum(v.y), warp_sum(v.z), warp_sum(v.w));
}

__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = threadIdx.x < (blockDim.x >> 5) ? part[threadIdx.x] : 0.f;
  if (threadIdx.x < 32) {
    t = warp_sum(t);
    if (threadIdx.x == 0) part[0] = t;
  }
  __syncthreads();
  return part[0];
}

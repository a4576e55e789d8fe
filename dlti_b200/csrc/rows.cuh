// Row-wise building blocks of the layer-stack kernels (stack.cu, streams.cu, latent.cu): typed and accumulator loads of
// projection rows, 16-byte pieces, block sums, where the rows of a sequence lie in a step.
//
// T is the activation type (bf16 or fp32). Kernels that consume a projection exist twice: from its T-typed output, and
// (ACC) straight from the fp32 accumulator of the decode GEMM, each value rounded to T as the stand-alone finish pass would
// and the accumulator left zero for the next GEMM. Every accumulator element is read by exactly one thread.
#pragma once
#include "common.cuh"

namespace {

template <typename T>
__device__ __forceinline__ float round_to(float v) { return Cvt<T>::to_f(Cvt<T>::from_f(v)); }

// element i of a projection row
template <typename T, bool ACC>
__device__ __forceinline__ float take(const void* row, long long i) {
  if constexpr (ACC) {
    float* p = const_cast<float*>(reinterpret_cast<const float*>(row)) + i;
    const float v = *p;
    *p = 0.f;
    return round_to<T>(v);
  } else {
    return Cvt<T>::to_f(reinterpret_cast<const T*>(row)[i]);
  }
}
// elements i, i+1 (i even, rows 16-byte aligned)
template <typename T, bool ACC>
__device__ __forceinline__ float2 take2(const void* row, long long i) {
  if constexpr (ACC) {
    float2* p = reinterpret_cast<float2*>(const_cast<float*>(reinterpret_cast<const float*>(row)) + i);
    const float2 v = *p;
    *p = make_float2(0.f, 0.f);
    return make_float2(round_to<T>(v.x), round_to<T>(v.y));
  } else if constexpr (sizeof(T) == 2) {
    return Cvt<T>::unpack2(*reinterpret_cast<const uint32_t*>(reinterpret_cast<const T*>(row) + i));
  } else {
    return *reinterpret_cast<const float2*>(reinterpret_cast<const float*>(row) + i);
  }
}
template <typename T>
__device__ __forceinline__ void put2(T* row, long long i, float a, float b) {
  if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(row + i) = Cvt<T>::pack2(a, b);
  else *reinterpret_cast<float2*>(row + i) = make_float2(a, b);
}

// N (2, 4 or 8) consecutive elements at an offset that is a multiple of N
template <typename T, bool ACC, int N>
__device__ __forceinline__ void take_n(const void* row, long long i, float (&f)[N]) {
  if constexpr (ACC) {
    float* p = const_cast<float*>(reinterpret_cast<const float*>(row)) + i;
    if constexpr (N == 2) {
      const float2 v = *reinterpret_cast<float2*>(p);
      *reinterpret_cast<float2*>(p) = make_float2(0.f, 0.f);
      f[0] = round_to<T>(v.x); f[1] = round_to<T>(v.y);
    } else {
#pragma unroll
      for (int j = 0; j < N / 4; ++j) {
        const float4 v = reinterpret_cast<float4*>(p)[j];
        reinterpret_cast<float4*>(p)[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        f[4 * j] = round_to<T>(v.x); f[4 * j + 1] = round_to<T>(v.y); f[4 * j + 2] = round_to<T>(v.z); f[4 * j + 3] = round_to<T>(v.w);
      }
    }
  } else if constexpr (sizeof(T) == 2) {
    const T* p = reinterpret_cast<const T*>(row) + i;
    uint32_t u[N / 2];
    if constexpr (N == 2) u[0] = *reinterpret_cast<const uint32_t*>(p);
    else if constexpr (N == 4) *reinterpret_cast<uint2*>(u) = *reinterpret_cast<const uint2*>(p);
    else *reinterpret_cast<uint4*>(u) = *reinterpret_cast<const uint4*>(p);
#pragma unroll
    for (int j = 0; j < N / 2; ++j) {
      const float2 v = Cvt<T>::unpack2(u[j]);
      f[2 * j] = v.x; f[2 * j + 1] = v.y;
    }
  } else {
#pragma unroll
    for (int j = 0; j < N; ++j) f[j] = reinterpret_cast<const float*>(row)[i + j];
  }
}
template <typename T, int N>
__device__ __forceinline__ void put_n(T* p, const float (&f)[N]) {
  if constexpr (sizeof(T) == 2) {
    uint32_t u[N / 2];
#pragma unroll
    for (int j = 0; j < N / 2; ++j) u[j] = Cvt<T>::pack2(f[2 * j], f[2 * j + 1]);
    if constexpr (N == 2) *reinterpret_cast<uint32_t*>(p) = u[0];
    else if constexpr (N == 4) *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(u);
    else *reinterpret_cast<uint4*>(p) = *reinterpret_cast<uint4*>(u);
  } else {
#pragma unroll
    for (int j = 0; j < N; ++j) p[j] = Cvt<T>::from_f(f[j]);
  }
}
__device__ __forceinline__ void ld8(const float* p, float (&f)[8]) {
  *reinterpret_cast<float4*>(f) = reinterpret_cast<const float4*>(p)[0];
  *reinterpret_cast<float4*>(f + 4) = reinterpret_cast<const float4*>(p)[1];
}
__device__ __forceinline__ void st8(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = *reinterpret_cast<const float4*>(f);
  reinterpret_cast<float4*>(p)[1] = *reinterpret_cast<const float4*>(f + 4);
}

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  return warp_sum(l < nw ? red[l] : 0.f);
}
__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }    // 16-bit outputs
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

// sequence s of a step: the first nd sequences are single rows, sequence nd + i has the rows nd + cu[i] ... nd + cu[i + 1]
__device__ __forceinline__ void seq_rows(const int* cu, const int* ctx, int nd, int s, long long& row0, int& n, int& start) {
  if (s < nd) {
    row0 = s;
    n = 1;
  } else {
    row0 = nd + cu[s - nd];
    n = cu[s - nd + 1] - cu[s - nd];
  }
  start = ctx[s] - n;
}

inline int grid_for(long long total, int block) {
  long long g = (total + block - 1) / block;
  const long long cap = (long long)dlti_num_sms() * 16;
  return (int)(g < 1 ? 1 : (g > cap ? cap : g));
}

}  // namespace

#define DISPATCH_T(dtype, CALL)                                      \
  do {                                                               \
    if ((dtype) == DLTI_BF16) { using T = __nv_bfloat16; CALL; }     \
    else if ((dtype) == DLTI_FP32) { using T = float; CALL; }        \
    else return DLTI_ERR_UNSUPPORTED;                                \
  } while (0)

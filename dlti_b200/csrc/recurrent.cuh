// Parts shared by the recurrences over the rows of a step (recurrent.cu, delta.cu): where a sequence's rows lie, decays, the
// renewal of a convolution's state. Params: nd, cu, ctx, sslot and the conv_* fields of ScanParams.
#pragma once
#include "common.cuh"

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// exp(x) of a decay. Near 1 the rounding of exp itself repeats at every token and adds up over a long memory; 1 + expm1
// rounds once.
__device__ __forceinline__ float decay_of(float x) { return x > -0.5f ? 1.f + expm1f(x) : expf(x); }

// sequence s: the first nd sequences are single rows, sequence nd + i has the rows nd + cu[i] ... nd + cu[i + 1]
template <typename Params>
__device__ __forceinline__ void seq_rows(const Params& p, int s, long long& row0, int& n, int& start) {
  if (s < p.nd) {
    row0 = s;
    n = 1;
  } else {
    row0 = p.nd + p.cu[s - p.nd];
    n = p.cu[s - p.nd + 1] - p.cu[s - p.nd];
  }
  start = p.ctx[s] - n;
}

// Shift the convolution inputs of one sequence: entry j becomes the input at position end - conv_rows + j. A thread
// owns whole channels and walks j upwards, so reading an old entry (always at a higher index) is safe.
template <typename T, typename Params>
__device__ __forceinline__ void conv_tail(const Params& p, int s, int part, int parts) {
  const int slot = p.sslot[s];
  if (slot < 0) return;
  long long row0;
  int n, start;
  seq_rows(p, s, row0, n, start);
  const T* src = reinterpret_cast<const T*>(p.conv_src);
  T* st = reinterpret_cast<T*>(p.conv_state) + (long long)slot * p.conv_rows * p.conv_C;
  for (int c = part * blockDim.x + threadIdx.x; c < p.conv_C; c += parts * blockDim.x)
    for (int j = 0; j < p.conv_rows; ++j) {
      const int q = n - p.conv_rows + j;
      T v = Cvt<T>::from_f(0.f);
      if (q >= 0) v = src[(row0 + q) * p.conv_ld + p.conv_col + c];
      else if (start > 0) v = st[(long long)(q + p.conv_rows) * p.conv_C + c];
      st[(long long)j * p.conv_C + c] = v;
    }
}

// RMS norms on the sublayer inputs of a model with one fp32 residual x:
//
//   prenorm_between  x += mult * y (or mult * norm(y) * post), x += embedding, h = norm(x) * pre (or a rounded copy): y is a sublayer's
//                    output, its decode GEMM's accumulator, or the sum that a mixture of experts leaves to its consumer (rows of the
//                    chosen experts times their weights, plus the shared expert times the token's share of it)
//   token_gate       gelu(u) times a part of the token's row of a table
//
// One CTA per row; the row stays in registers between the sums.
#include <initializer_list>

#include "rows.cuh"

namespace {

struct Between {
  float* x;
  const void* y; long long y_ld;                           // sublayer output or shared expert (null: none)
  const void* rows; long long r_ld;                        // outputs of the chosen experts, top rows a token (null: no mixture)
  const float* weights; int top;
  const float* share;                                      // factor of y per token (null: one)
  int* counts; int ncounts;                                // router counters to clear
  float mult;
  const float* post;                                       // norm weights of what is added (null: no norm)
  const long long* ids; const void* table; long long vocab; float scale;      // embedding to add (null: none)
  int fresh;                                               // x starts as zero
  const float* pre; void* h; long long h_ld;               // pre null: h = x; h null: nothing is read next
  int d; float eps;
};

template <typename T, bool ACC, int W>
__device__ __forceinline__ void piece(const void* row, int c, float (&f)[W]) {
  if constexpr (W == 1) f[0] = take<T, ACC>(row, c);
  else take_n<T, ACC, W>(row, c, f);
}
template <int W>
__device__ __forceinline__ void piece_f32(const float* p, float (&f)[W]) {
  if constexpr (W == 8) ld8(p, f);
  else f[0] = p[0];
}

template <typename T, bool ACC, int W, int VPT, int THREADS>
__global__ void __launch_bounds__(THREADS) prenorm_between_kernel(const Between p) {
  __shared__ float red[32];
  float wv[VPT][W];
  const bool norm = p.pre != nullptr;
  if (norm) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {                        // weights never change: they may come before the wait
      const int c = (threadIdx.x + i * THREADS) * W;
      if (c < p.d) piece_f32<W>(p.pre + c, wv[i]);
    }
  }
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  if (p.counts && t == 0)
    for (int i = threadIdx.x; i < p.ncounts; i += THREADS) p.counts[i] = 0;
  float* xr = p.x + t * p.d;
  float f[VPT][W], x[VPT][W];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * THREADS) * W;
#pragma unroll
    for (int j = 0; j < W; ++j) f[i][j] = x[i][j] = 0.f;
    if (c < p.d) {
      if (!p.fresh) piece_f32<W>(xr + c, x[i]);
      if (p.y) piece<T, ACC, W>(reinterpret_cast<const uint8_t*>(p.y) + t * p.y_ld * (ACC ? 4 : sizeof(T)), c, f[i]);
    }
  }
  if (p.share) {
    const float s = p.share[t];
#pragma unroll
    for (int i = 0; i < VPT; ++i)
#pragma unroll
      for (int j = 0; j < W; ++j) f[i][j] *= s;
  }
  if (p.rows) {
    const T* er = reinterpret_cast<const T*>(p.rows) + t * p.top * p.r_ld;
#pragma unroll 4
    for (int k = 0; k < p.top; ++k) {
      const float w = p.weights[t * p.top + k];
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = (threadIdx.x + i * THREADS) * W;
        if (c < p.d) {
          float e[W];
          piece<T, false, W>(er + k * p.r_ld, c, e);
#pragma unroll
          for (int j = 0; j < W; ++j) f[i][j] = fmaf(w, e[j], f[i][j]);
        }
      }
    }
  }
  if (p.post) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i)
#pragma unroll
      for (int j = 0; j < W; ++j) ss += f[i][j] * f[i][j];
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)p.d + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * THREADS) * W;
      if (c < p.d) {
        float w[W];
        piece_f32<W>(p.post + c, w);
#pragma unroll
        for (int j = 0; j < W; ++j) f[i][j] *= r * w[j];
      }
    }
  }
  const long long id = p.ids ? p.ids[t] : -1;
  const bool add = id >= 0 && id < p.vocab;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * THREADS) * W;
    if (c < p.d) {
#pragma unroll
      for (int j = 0; j < W; ++j) x[i][j] = fmaf(p.mult, f[i][j], x[i][j]);
      if (add) {
        float e[W];
        piece<T, false, W>(reinterpret_cast<const T*>(p.table) + id * p.d, c, e);
#pragma unroll
        for (int j = 0; j < W; ++j) x[i][j] = fmaf(p.scale, e[j], x[i][j]);
      }
      if constexpr (W == 8) st8(xr + c, x[i]);
      else xr[c] = x[i][0];
#pragma unroll
      for (int j = 0; j < W; ++j) ss += x[i][j] * x[i][j];
    }
  }
  if (!p.h) return;
  const float r = norm ? 1.f / sqrtf(block_sum(ss, red) / (float)p.d + p.eps) : 1.f;
  T* hr = reinterpret_cast<T*>(p.h) + t * p.h_ld;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * THREADS) * W;
    if (c < p.d) {
      if (norm)
#pragma unroll
        for (int j = 0; j < W; ++j) x[i][j] *= r * wv[i][j];
      if constexpr (W == 1) hr[c] = Cvt<T>::from_f(x[i][0]);
      else put_n(hr + c, x[i]);
    }
  }
}

__device__ __forceinline__ float gelu_tanh(float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

template <typename T, bool ACC, int W>
__global__ void __launch_bounds__(128) token_gate_kernel(const void* __restrict__ u, long long u_ld, const long long* __restrict__ ids,
                                                         const T* __restrict__ table, long long t_ld, long long vocab, int col, int n,
                                                         T* __restrict__ h, long long h_ld, long long tokens) {
  griddep_wait();
  griddep_launch();
  const int per = n / W;
  const long long total = tokens * per;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / per, id = ids[t];
    const int c = (int)(i - t * per) * W;
    float a[W], e[W];
    piece<T, ACC, W>(reinterpret_cast<const uint8_t*>(u) + t * u_ld * (ACC ? 4 : sizeof(T)), c, a);
    if (id >= 0 && id < vocab) {
      piece<T, false, W>(table + id * t_ld + col, c, e);
    } else {
#pragma unroll
      for (int j = 0; j < W; ++j) e[j] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < W; ++j) a[j] = gelu_tanh(a[j]) * e[j];
    if constexpr (W == 1) h[t * h_ld + c] = Cvt<T>::from_f(a[0]);
    else put_n(h + t * h_ld + c, a);
  }
}

bool aligned16(std::initializer_list<const void*> ps) {
  uintptr_t u = 0;
  for (const void* p : ps) u |= reinterpret_cast<uintptr_t>(p);
  return (u & 15) == 0;
}

template <typename T, bool ACC>
int between(const Between& p, long long tokens, cudaStream_t st) {
#define PB_CASE(W, V, TH)                                                                                                               \
  if (p.d <= W * V * TH) {                                                                                                              \
    DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, prenorm_between_kernel<T, ACC, W, V, TH>, dim3((unsigned)tokens), dim3(TH), 0, st, p));      \
    dlti_count_launch();                                                                                                                \
    return 0;                                                                                                                           \
  }
  if constexpr (sizeof(T) == 2) {
    if (((p.d | p.y_ld | p.r_ld | p.h_ld) & 7) == 0 && aligned16({p.x, p.y, p.rows, p.post, p.table, p.pre, p.h})) {
      PB_CASE(8, 1, 128) PB_CASE(8, 1, 256) PB_CASE(8, 1, 512) PB_CASE(8, 2, 512)
    }
  }
  PB_CASE(1, 1, 256) PB_CASE(1, 4, 256) PB_CASE(1, 16, 256) PB_CASE(1, 32, 512)
#undef PB_CASE
  dlti_set_error("prenorm_between: rows of up to 16384 elements");
  return DLTI_ERR_TOO_LARGE;
}

}  // namespace

// see Between; acc: y is the decode GEMM's accumulator (zero on return)
DLTI_API int dlti_prenorm_between(float* x, const void* y, long long y_ld, const void* rows, long long r_ld, const float* weights, int top,
                                  const float* share, int* counts, int ncounts, float mult, const float* post, const long long* ids,
                                  const void* table, long long vocab, float scale, int fresh, const float* pre, void* h, long long h_ld,
                                  long long tokens, int d, float eps, int acc, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if ((rows && (!weights || top < 1)) || (pre && !h) || (ids && !table) || (share && !y) || (acc && !y) || d < 1) return DLTI_ERR_BAD_ARG;
  const Between p{x, y, y_ld, rows, r_ld, weights, top, share, counts, ncounts, mult, post, ids, table, vocab, scale, fresh, pre, h, h_ld, d, eps};
  if (acc) DISPATCH_T(dtype, return (between<T, true>(p, tokens, st)));
  DISPATCH_T(dtype, return (between<T, false>(p, tokens, st)));
}

// h[t, 0 .. n) = gelu(u[t, c]) * table[ids[t], col + c]; acc: u is the decode GEMM's accumulator (zero on return)
DLTI_API int dlti_token_gate(const void* u, long long u_ld, const long long* ids, const void* table, long long t_ld, long long vocab, int col,
                             int n, void* h, long long h_ld, long long tokens, int acc, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (n < 1 || col < 0 || col + n > t_ld) return DLTI_ERR_BAD_ARG;
  using B = __nv_bfloat16;
#define TG_LAUNCH(T, AC, W)                                                                                                            \
  DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, token_gate_kernel<T, AC, W>, dim3(grid_for(tokens * (n / W), 128)), dim3(128), 0, st, u, u_ld, ids, \
                                  (const T*)table, t_ld, vocab, col, n, (T*)h, h_ld, tokens))
  if (dtype == DLTI_BF16 && ((n | col) & 7) == 0 && ((u_ld | t_ld | h_ld) & 7) == 0 && aligned16({u, table, h})) {
    if (acc) TG_LAUNCH(B, true, 8);
    else TG_LAUNCH(B, false, 8);
  } else if (acc) {
    DISPATCH_T(dtype, TG_LAUNCH(T, true, 1));
  } else {
    DISPATCH_T(dtype, TG_LAUNCH(T, false, 1));
  }
#undef TG_LAUNCH
  dlti_count_launch();
  return 0;
}

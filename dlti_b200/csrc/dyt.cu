// Dynamic tanh norms, tanh(alpha x) * w + b, around the sublayers of a model with one fp32 residual x:
//
//   tanh_embed     x = scale * table[ids],  h = pre(x)
//   tanh_between   x += post(y),  h = pre(x): y is a sublayer's output, its decode GEMM's accumulator, or the sum that a mixture
//                  of experts leaves to its consumer (rows of the chosen experts times their weights, plus the shared expert)
//   tanh_rows      h = norm(x[idx])
//
// There is no reduction over a row: every kernel is elementwise in pieces of W elements (8 where sizes and pitches allow it).
#include <initializer_list>

#include "rows.cuh"

namespace {

struct Norm { const float *alpha, *w, *b; };

__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <typename T, int W>
__device__ __forceinline__ void norm_piece(const Norm& n, float alpha, int c, const float (&x)[W], float (&out)[W]) {
  float w[W], b[W];
  if constexpr (W == 8) {
    ld8(n.w + c, w);
    ld8(n.b + c, b);
  } else {
#pragma unroll
    for (int j = 0; j < W; ++j) { w[j] = n.w[c + j]; b[j] = n.b[c + j]; }
  }
  if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int j = 0; j < W; ++j) out[j] = fmaf(tanhf(alpha * x[j]), w[j], b[j]);
  } else {                                                 // tanh z = 1 - 2 / (1 + e^(2 z)): absolute error about 1e-7
    const float a = 2.f * 1.4426950408889634f * alpha;
#pragma unroll
    for (int j = 0; j < W; ++j) out[j] = fmaf(-2.f * w[j], rcp_approx(1.f + ex2_approx(a * x[j])), w[j] + b[j]);
  }
}
template <typename T, bool ACC, int W>
__device__ __forceinline__ void load_piece(const void* row, int c, float (&f)[W]) {
  if constexpr (W == 1) f[0] = take<T, ACC>(row, c);
  else take_n<T, ACC, W>(row, c, f);
}
template <typename T, int W>
__device__ __forceinline__ void store_piece(T* p, const float (&f)[W]) {
  if constexpr (W == 1) *p = Cvt<T>::from_f(f[0]);
  else put_n(p, f);
}
template <int W>
__device__ __forceinline__ void x_load(const float* p, float (&f)[W]) {
  if constexpr (W == 8) ld8(p, f);
  else f[0] = p[0];
}
template <int W>
__device__ __forceinline__ void x_store(float* p, const float (&f)[W]) {
  if constexpr (W == 8) st8(p, f);
  else p[0] = f[0];
}

template <typename T, int W>
__global__ void __launch_bounds__(128) tanh_embed_kernel(const long long* __restrict__ ids, const T* __restrict__ table, long long vocab,
                                                         float scale, Norm pre, float* __restrict__ x, T* __restrict__ h, long long h_ld, int d) {
  griddep_wait();
  griddep_launch();
  const int c = (blockIdx.y * 128 + threadIdx.x) * W;
  if (c >= d) return;
  const long long t = blockIdx.x, id = ids[t];
  float f[W], o[W];
  if (id >= 0 && id < vocab) {
    load_piece<T, false, W>(table + id * d, c, f);
  } else {
#pragma unroll
    for (int j = 0; j < W; ++j) f[j] = 0.f;
  }
#pragma unroll
  for (int j = 0; j < W; ++j) f[j] *= scale;
  x_store<W>(x + t * d + c, f);
  norm_piece<T, W>(pre, *pre.alpha, c, f, o);
  store_piece<T, W>(h + t * h_ld + c, o);
}

struct Between {
  float* x;
  const void* y; long long y_ld;                           // sublayer output or shared expert (null: none)
  const void* rows; long long r_ld;                        // outputs of the chosen experts, top rows a token (null: no mixture)
  const float* weights; int top;
  int* counts; int ncounts;                                // router counters to clear
  Norm post, pre;                                          // pre.w null: nothing is read next
  void* h; long long h_ld;
  int d;
};
constexpr int TB_ROWS = 2;                                 // tokens per thread: the norm vectors are loaded once
template <typename T, bool ACC, int W, int ROWS>
__global__ void __launch_bounds__(128) tanh_between_kernel(const Between p, long long tokens) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * W;
  const bool on = c < p.d;
  griddep_wait();
  griddep_launch();
  if (p.counts && blockIdx.x == 0 && blockIdx.y == 0)
    for (int i = threadIdx.x; i < p.ncounts; i += 128) p.counts[i] = 0;
  if (!on) return;
  const float a_post = *p.post.alpha, a_pre = p.pre.w ? *p.pre.alpha : 0.f;
  const long long t0 = (long long)blockIdx.x * ROWS;
  float f[ROWS][W], xv[ROWS][W];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const long long t = t0 + r;
    if (t >= tokens) break;
    x_load<W>(p.x + t * p.d + c, xv[r]);
    if (p.y) {
      load_piece<T, ACC, W>(reinterpret_cast<const uint8_t*>(p.y) + t * p.y_ld * (ACC ? 4 : sizeof(T)), c, f[r]);
    } else {
#pragma unroll
      for (int j = 0; j < W; ++j) f[r][j] = 0.f;
    }
  }
  if (p.rows) {
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const long long t = t0 + r;
      if (t >= tokens) break;
      const T* er = reinterpret_cast<const T*>(p.rows) + t * p.top * p.r_ld;
#pragma unroll 4
      for (int k = 0; k < p.top; ++k) {
        float e[W];
        load_piece<T, false, W>(er + k * p.r_ld, c, e);
        const float w = p.weights[t * p.top + k];
#pragma unroll
        for (int j = 0; j < W; ++j) f[r][j] = fmaf(w, e[j], f[r][j]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const long long t = t0 + r;
    if (t >= tokens) break;
    float o[W];
    norm_piece<T, W>(p.post, a_post, c, f[r], o);
#pragma unroll
    for (int j = 0; j < W; ++j) xv[r][j] += o[j];
    x_store<W>(p.x + t * p.d + c, xv[r]);
    if (p.pre.w) {
      norm_piece<T, W>(p.pre, a_pre, c, xv[r], o);
      store_piece<T, W>(reinterpret_cast<T*>(p.h) + t * p.h_ld + c, o);
    }
  }
}

template <typename T, int W>
__global__ void __launch_bounds__(128) tanh_rows_kernel(const float* __restrict__ x, const long long* __restrict__ idx, Norm n,
                                                        T* __restrict__ h, long long h_ld, int d) {
  griddep_wait();
  griddep_launch();
  const int c = (blockIdx.y * 128 + threadIdx.x) * W;
  if (c >= d) return;
  const long long t = blockIdx.x;
  float f[W], o[W];
  x_load<W>(x + (idx ? idx[t] : t) * d + c, f);
  norm_piece<T, W>(n, *n.alpha, c, f, o);
  store_piece<T, W>(h + t * h_ld + c, o);
}

bool aligned16(std::initializer_list<const void*> ps) {
  uintptr_t u = 0;
  for (const void* p : ps) u |= reinterpret_cast<uintptr_t>(p);
  return (u & 15) == 0;
}
dim3 piece_grid(long long rows, int d, int W) { return dim3((unsigned)rows, (d + 128 * W - 1) / (128 * W)); }

template <typename T, bool ACC, int W>
int between(const Between& p, long long tokens, cudaStream_t st) {
  // several tokens a thread once that still fills the GPU
  const bool many = W == 8 && tokens * p.d >= (long long)dlti_num_sms() * 2048 * 8 * TB_ROWS / 2;
  auto kern = many ? tanh_between_kernel<T, ACC, W, TB_ROWS> : tanh_between_kernel<T, ACC, W, 1>;
  DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, kern, piece_grid(many ? (tokens + TB_ROWS - 1) / TB_ROWS : tokens, p.d, W), dim3(128), 0, st, p, tokens));
  dlti_count_launch();
  return 0;
}

}  // namespace

// norms: (alpha [1], w [d], b [d]); h [tokens, >= d] in dtype
DLTI_API int dlti_tanh_embed(const long long* ids, const void* table, long long vocab, float scale, const float* alpha, const float* w,
                             const float* b, float* x, void* h, long long h_ld, long long tokens, int d, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  const Norm n{alpha, w, b};
  using B = __nv_bfloat16;
  if (dtype == DLTI_BF16 && d % 8 == 0 && h_ld % 8 == 0 && aligned16({table, w, b, x, h})) {
    DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, tanh_embed_kernel<B, 8>, piece_grid(tokens, d, 8), dim3(128), 0, st, ids, (const B*)table, vocab, scale, n,
                                    x, (B*)h, h_ld, d));
  } else {
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, tanh_embed_kernel<T, 1>, piece_grid(tokens, d, 1), dim3(128), 0, st, ids,
                                                      (const T*)table, vocab, scale, n, x, (T*)h, h_ld, d)));
  }
  dlti_count_launch();
  return 0;
}

// y, rows / weights / counts and the second norm with h may be null; acc: y is the decode GEMM's accumulator (zero on return)
DLTI_API int dlti_tanh_between(float* x, const void* y, long long y_ld, const void* rows, long long r_ld, const float* weights, int top,
                               int* counts, int ncounts, const float* alpha1, const float* w1, const float* b1, const float* alpha2,
                               const float* w2, const float* b2, void* h, long long h_ld, long long tokens, int d, int acc, int dtype,
                               cudaStream_t st) {
  if (tokens <= 0) return 0;
  if ((rows && (!weights || top < 1)) || (w2 && !h)) return DLTI_ERR_BAD_ARG;
  const Between p{x, y, y_ld, rows, r_ld, weights, top, counts, ncounts, {alpha1, w1, b1}, {alpha2, w2, b2}, h, h_ld, d};
  using B = __nv_bfloat16;
  if (dtype == DLTI_BF16 && ((d | y_ld | r_ld | h_ld) & 7) == 0 && aligned16({x, y, rows, w1, b1, w2, b2, h}))
    return acc ? between<B, true, 8>(p, tokens, st) : between<B, false, 8>(p, tokens, st);
  if (acc) DISPATCH_T(dtype, return (between<T, true, 1>(p, tokens, st)));
  DISPATCH_T(dtype, return (between<T, false, 1>(p, tokens, st)));
}

DLTI_API int dlti_tanh_rows(const float* x, const long long* idx, const float* alpha, const float* w, const float* b, void* h, long long h_ld,
                            long long rows, int d, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  const Norm n{alpha, w, b};
  using B = __nv_bfloat16;
  if (dtype == DLTI_BF16 && d % 8 == 0 && h_ld % 8 == 0 && aligned16({x, w, b, h})) {
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, tanh_rows_kernel<B, 8>, piece_grid(rows, d, 8), dim3(128), 0, st, x, idx, n, (B*)h, h_ld, d));
  } else {
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, tanh_rows_kernel<T, 1>, piece_grid(rows, d, 1), dim3(128), 0, st, x, idx, n, (T*)h, h_ld,
                                                      d)));
  }
  dlti_count_launch();
  return 0;
}

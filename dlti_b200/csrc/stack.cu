// Row-wise kernels of the layer-stack models (models/stack.py): fp32 residual stream, norms on the sublayer outputs,
// per-head query/key norm + rotary + paged-cache write, squared relu, gated norms, short causal convolutions.
//
// T is the activation type (bf16 or fp32); residual, norms, gates and rotations are fp32 in either case. Kernels that
// consume a projection exist twice: from its T-typed output, and (ACC) straight from the fp32 accumulator of the
// decode GEMM, each value rounded to T as the stand-alone finish pass would and the accumulator left zero for the next
// GEMM. Every accumulator element is read by exactly one thread.
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

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  return warp_sum(l < nw ? red[l] : 0.f);
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

// x[t] = table[ids[t]] (fp32 residual) and, for 16-bit activations, the same row as the first GEMM's input
template <typename T>
__global__ void embed_rows_kernel(const long long* __restrict__ ids, const T* __restrict__ table, float* __restrict__ x,
                                  T* __restrict__ xa, long long xa_ld, long long tokens, int d, long long vocab) {
  griddep_wait();
  griddep_launch();
  const long long total = tokens * d;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / d;
    const int c = (int)(i - t * d);
    const long long id = ids[t];
    const T v = (id >= 0 && id < vocab) ? table[id * d + c] : Cvt<T>::from_f(0.f);
    x[i] = Cvt<T>::to_f(v);
    if (xa) xa[t * xa_ld + c] = v;
  }
}

// out = acc (fp32), acc = 0
__global__ void take_rows_kernel(float* __restrict__ acc, float* __restrict__ out, long long vec) {
  griddep_wait();
  griddep_launch();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < vec; i += (long long)gridDim.x * blockDim.x) {
    reinterpret_cast<float4*>(out)[i] = reinterpret_cast<float4*>(acc)[i];
    reinterpret_cast<float4*>(acc)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
}

// x += norm(y) * w (or * (1 + w)); xa = T(x). One CTA per row; the row of y stays in registers.
constexpr int PN_THREADS = 256;
template <typename T, bool ACC, int PAIRS>
__global__ void __launch_bounds__(PN_THREADS) post_norm_add_kernel(const void* __restrict__ y, long long y_ld, float* __restrict__ x,
                                                                  const float* __restrict__ w, T* __restrict__ xa,
                                                                  long long xa_ld, int d, float eps, float one) {
  __shared__ float red[32];
  griddep_wait();
  griddep_launch();
  const long long row = blockIdx.x;
  const void* yr = reinterpret_cast<const uint8_t*>(y) + row * y_ld * (ACC ? 4 : sizeof(T));
  float* xr = x + row * d;
  float2 v[PAIRS];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < PAIRS; ++i) {
    const int c = 2 * (threadIdx.x + i * PN_THREADS);
    v[i] = make_float2(0.f, 0.f);
    if (c + 1 < d) v[i] = take2<T, ACC>(yr, c);
    else if (c < d) v[i].x = take<T, ACC>(yr, c);
    ss += v[i].x * v[i].x + v[i].y * v[i].y;
  }
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)d + eps);
#pragma unroll
  for (int i = 0; i < PAIRS; ++i) {
    const int c = 2 * (threadIdx.x + i * PN_THREADS);
    if (c < d) {
      const float a = xr[c] + v[i].x * r * (one + w[c]);
      xr[c] = a;
      if (xa) xa[row * xa_ld + c] = Cvt<T>::from_f(a);
    }
    if (c + 1 < d) {
      const float a = xr[c + 1] + v[i].y * r * (one + w[c + 1]);
      xr[c + 1] = a;
      if (xa) xa[row * xa_ld + c + 1] = Cvt<T>::from_f(a);
    }
  }
}

// out[i] = norm(x[idx[i]]) * w (or * (1 + w))
template <typename T>
__global__ void __launch_bounds__(PN_THREADS) rms_rows_kernel(const float* __restrict__ x, const long long* __restrict__ idx,
                                                             const float* __restrict__ w, T* __restrict__ out,
                                                             long long out_ld, int d, float eps, float one) {
  __shared__ float red[32];
  griddep_wait();
  griddep_launch();
  const float* xr = x + (idx ? idx[blockIdx.x] : (long long)blockIdx.x) * d;
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += PN_THREADS) ss += xr[c] * xr[c];
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)d + eps);
  T* o = out + (long long)blockIdx.x * out_ld;
  for (int c = threadIdx.x; c < d; c += PN_THREADS) o[c] = Cvt<T>::from_f(xr[c] * r * (one + w[c]));
}

// h = relu(u)^2, columns in pairs (row pitches are even)
template <typename T, bool ACC>
__global__ void relu2_kernel(const void* __restrict__ u, long long u_ld, T* __restrict__ h, long long h_ld, long long rows, int ff) {
  griddep_wait();
  griddep_launch();
  const int pairs = (ff + 1) >> 1;
  const long long total = rows * pairs;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / pairs;
    const int c = 2 * (int)(i - t * pairs);
    const void* ur = reinterpret_cast<const uint8_t*>(u) + t * u_ld * (ACC ? 4 : sizeof(T));
    float2 v;
    if (c + 1 < ff) {
      v = take2<T, ACC>(ur, c);
      v.x = fmaxf(v.x, 0.f);
      v.y = fmaxf(v.y, 0.f);
      put2(h + t * h_ld, c, v.x * v.x, v.y * v.y);
    } else {
      const float a = fmaxf(take<T, ACC>(ur, c), 0.f);
      h[t * h_ld + c] = Cvt<T>::from_f(a * a);
    }
  }
}
// the same, 8 columns per thread (16-bit, both pitches and ff multiples of 8)
template <typename T>
__global__ void relu2_vec_kernel(const T* __restrict__ u, long long u_ld, T* __restrict__ h, long long h_ld, long long rows, int ff) {
  const int vec = ff >> 3;
  const long long total = rows * vec;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / vec;
    const int c = 8 * (int)(i - t * vec);
    int4 v = *reinterpret_cast<const int4*>(u + t * u_ld + c);
    uint32_t* p = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float2 f = Cvt<T>::unpack2(p[j]);
      f.x = fmaxf(f.x, 0.f);
      f.y = fmaxf(f.y, 0.f);
      p[j] = Cvt<T>::pack2(f.x * f.x, f.y * f.y);
    }
    *reinterpret_cast<int4*>(h + t * h_ld + c) = v;
  }
}

// Norm of a mixer output in `groups` equal parts with a multiplicative gate.
//   GATE_FIRST:  out = norm(y * silu(g)) * w          (Mamba-2)
//   otherwise:   out = norm(y) * w * sigmoid(g)       (lightning attention)
// One CTA per row, one warp per group in turn; a group is passed twice (second time from L1).
template <typename T, bool GATE_FIRST, bool ACC>
__global__ void __launch_bounds__(256) gated_norm_kernel(const T* __restrict__ y, long long y_ld, const void* __restrict__ gate,
                                                         long long g_ld, const float* __restrict__ w, T* __restrict__ out,
                                                         long long o_ld, int n, int groups, float eps) {
  __shared__ float red[32];
  extern __shared__ float row_s[];          // the gated row (GATE_FIRST) or the gate factors
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  const T* yr = y + t * y_ld;
  const void* gr = reinterpret_cast<const uint8_t*>(gate) + t * g_ld * (ACC ? 4 : sizeof(T));
  const int gs = n / groups;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    const float g = take<T, ACC>(gr, c);
    row_s[c] = GATE_FIRST ? Cvt<T>::to_f(yr[c]) * silu_f(g) : sigmoid_f(g);
  }
  __syncthreads();
  if (groups == 1) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float v = GATE_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]);
      ss += v * v;
    }
    ss = block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / (float)n + eps);
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float v = (GATE_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]) * row_s[c]) * r * w[c];
      out[t * o_ld + c] = Cvt<T>::from_f(v);
    }
    return;
  }
  for (int g = threadIdx.x >> 5; g < groups; g += blockDim.x >> 5) {
    float ss = 0.f;
    for (int c = g * gs + (threadIdx.x & 31); c < (g + 1) * gs; c += 32) {
      const float v = GATE_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]);
      ss += v * v;
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)gs + eps);
    for (int c = g * gs + (threadIdx.x & 31); c < (g + 1) * gs; c += 32) {
      const float v = (GATE_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]) * row_s[c]) * r * w[c];
      out[t * o_ld + c] = Cvt<T>::from_f(v);
    }
  }
}

// Per-head norm + rotation of q and k, cache write of k and v, sigmoid of the head gates. One warp per (token, job):
// jobs = H query heads, G key heads, G value heads, then one job for all head gates. A layer on another layer's keys
// and values has no k / v jobs of its own; with a packed destination they copy the cached rows instead.
struct QkvParams {
  const void* proj; long long ld;         // merged projection rows
  int oq, ok, ov, og;                     // section columns (ok < 0: no own keys and values; og < 0: no gates)
  const float *qn, *kn; float eps;        // per-head norm weights (null: no norm)
  const int* pos; const float *cos_t, *sin_t; int rot; int interleaved;
  const long long* slots; void *kc, *vc; int kd, vd;       // cache row pitches of a head
  void* q; long long q_ld; int q_hd;                       // rotated queries: row pitch, head pitch
  void *kp, *vp;                                           // packed keys / values (row pitch q_ld, head pitch q_hd) or null
  float* gate;                                             // [tokens, H]
  long long tokens; int H, G, dim, vdim;
};
constexpr int QKV_MAXP = 8;               // pairs per lane: heads of up to 512
template <typename T, bool ACC>
__global__ void __launch_bounds__(256) qk_norm_rope_cache_kernel(const QkvParams p) {
  griddep_wait();
  griddep_launch();
  const bool own = p.ok >= 0, copy_kv = !own && p.kp;
  const int kvjobs = (own || copy_kv) ? 2 * p.G : 0;
  const int jobs = p.H + kvjobs + (p.og >= 0 ? 1 : 0);
  const int lane = threadIdx.x & 31;
  const long long total = p.tokens * jobs;
  for (long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5; w < total;
       w += ((long long)gridDim.x * blockDim.x) >> 5) {
    const long long t = w / jobs;
    const int job = (int)(w - t * jobs);
    const uint8_t* row = reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * (ACC ? 4 : sizeof(T));
    const long long slot = p.slots[t];
    if (job >= p.H + kvjobs) {
      for (int h = lane; h < p.H; h += 32) p.gate[t * p.H + h] = sigmoid_f(take<T, ACC>(row, p.og + h));
      continue;
    }
    if (job >= p.H + p.G) {                                          // a value head
      const int g = job - p.H - p.G;
      T* src = reinterpret_cast<T*>(p.vc) + (slot * p.G + g) * p.vd;
      T* pk = p.vp ? reinterpret_cast<T*>(p.vp) + t * p.q_ld + (long long)g * p.q_hd : nullptr;
      for (int c = lane; c < p.vdim; c += 32) {
        const T v = own ? Cvt<T>::from_f(take<T, ACC>(row, p.ov + g * p.vdim + c)) : (slot >= 0 ? src[c] : Cvt<T>::from_f(0.f));
        if (own && slot >= 0) src[c] = v;
        if (pk) pk[c] = v;
      }
      continue;
    }
    const bool is_q = job < p.H;
    const int head = is_q ? job : job - p.H;
    T* cache = reinterpret_cast<T*>(p.kc) + (slot * p.G + head) * p.kd;
    T* out = is_q ? reinterpret_cast<T*>(p.q) + t * p.q_ld + (long long)head * p.q_hd
                  : (p.kp ? reinterpret_cast<T*>(p.kp) + t * p.q_ld + (long long)head * p.q_hd : nullptr);
    if (!is_q && !own) {
      for (int c = lane; c < p.dim; c += 32) out[c] = slot >= 0 ? cache[c] : Cvt<T>::from_f(0.f);
      continue;
    }
    const int col = (is_q ? p.oq : p.ok) + head * p.dim;
    const float* nw = is_q ? p.qn : p.kn;
    const int half = p.rot >> 1, npair = half + ((p.dim - p.rot + 1) >> 1);
    float2 v[QKV_MAXP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < QKV_MAXP; ++i) {
      const int j = lane + 32 * i;
      v[i] = make_float2(0.f, 0.f);
      if (j < npair) {
        const int e0 = j < half ? (p.interleaved ? 2 * j : j) : p.rot + 2 * (j - half);
        const int e1 = j < half ? (p.interleaved ? 2 * j + 1 : j + half) : e0 + 1;
        if (e1 == e0 + 1 && e1 < p.dim && ((col + e0) & 1) == 0) {
          v[i] = take2<T, ACC>(row, col + e0);
        } else {
          v[i].x = take<T, ACC>(row, col + e0);
          if (e1 < p.dim) v[i].y = take<T, ACC>(row, col + e1);
        }
        ss += v[i].x * v[i].x + v[i].y * v[i].y;
      }
    }
    float r = 1.f;
    if (nw) r = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
    const int ps = p.pos[t];
#pragma unroll
    for (int i = 0; i < QKV_MAXP; ++i) {
      const int j = lane + 32 * i;
      if (j >= npair) continue;
      const int e0 = j < half ? (p.interleaved ? 2 * j : j) : p.rot + 2 * (j - half);
      const int e1 = j < half ? (p.interleaved ? 2 * j + 1 : j + half) : e0 + 1;
      float a = v[i].x * r, b = v[i].y * r;
      if (nw) {
        a *= nw[e0];
        if (e1 < p.dim) b *= nw[e1];
      }
      if (j < half) {
        const float c = p.cos_t[(long long)ps * half + j], s = p.sin_t[(long long)ps * half + j];
        const float u = a * c - b * s;
        b = b * c + a * s;
        a = u;
      }
      const T ta = Cvt<T>::from_f(a), tb = Cvt<T>::from_f(b);
      if (out) {
        out[e0] = ta;
        if (e1 < p.dim) out[e1] = tb;
      }
      if (!is_q && slot >= 0) {
        cache[e0] = ta;
        if (e1 < p.dim) cache[e1] = tb;
      }
    }
  }
}

// Causal convolution of `taps` per channel + silu over the rows of every sequence of a step. src = projection rows
// (channel 0 at column `col`); inputs from before the step come from conv_state [slots, taps - 1, C] (zero at position
// 0). ACC additionally leaves the rounded projection row in `raw` (columns raw0 .. raw0 + raw_n): the gate, the step
// sizes and the inputs that the state update needs afterwards.
struct ConvParams {
  const void* src; long long ld; int col, C, taps;
  const float *w, *b; int w_ld;                            // tap-major weights
  const void* state; const int *sslot, *rseq, *ctx, *cu; int nd;
  void* out; long long o_ld;
  void* raw; long long raw_ld; int raw_n;
  long long rows;
};
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
template <typename T>
__global__ void __launch_bounds__(256) short_conv_kernel(const ConvParams p) {
  griddep_wait();
  griddep_launch();
  const int pairs = (p.C + 1) >> 1;
  const long long total = p.rows * pairs;
  const T* src = reinterpret_cast<const T*>(p.src);
  const T* state = reinterpret_cast<const T*>(p.state);
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / pairs;
    const int c = 2 * (int)(i - t * pairs);
    const bool two = c + 1 < p.C;
    const int s = p.rseq[t];
    long long row0;
    int n, start;
    seq_rows(p.cu, p.ctx, p.nd, s, row0, n, start);
    const int local = (int)(t - row0);
    const int slot = p.sslot[s];
    float a0 = p.b[c], a1 = two ? p.b[c + 1] : 0.f;
    for (int k = 0; k < p.taps; ++k) {
      const int q = local - (p.taps - 1) + k;              // row of this tap relative to the step
      float x0 = 0.f, x1 = 0.f;
      if (q >= 0) {
        const T* r = src + (row0 + q) * p.ld + p.col + c;
        x0 = Cvt<T>::to_f(r[0]);
        if (two) x1 = Cvt<T>::to_f(r[1]);
      } else if (start > 0 && slot >= 0) {
        const T* r = state + ((long long)slot * (p.taps - 1) + q + p.taps - 1) * p.C + c;
        x0 = Cvt<T>::to_f(r[0]);
        if (two) x1 = Cvt<T>::to_f(r[1]);
      }
      a0 += p.w[(long long)k * p.w_ld + c] * x0;
      if (two) a1 += p.w[(long long)k * p.w_ld + c + 1] * x1;
    }
    T* o = reinterpret_cast<T*>(p.out) + t * p.o_ld + c;
    o[0] = Cvt<T>::from_f(silu_f(a0));
    if (two) o[1] = Cvt<T>::from_f(silu_f(a1));
  }
}
// decode rows only: the projection comes as the decode GEMM's accumulator
template <typename T>
__global__ void __launch_bounds__(256) short_conv_acc_kernel(const ConvParams p) {
  griddep_wait();
  griddep_launch();
  const int pairs = (p.raw_n + 1) >> 1;
  const long long total = p.rows * pairs;
  const T* state = reinterpret_cast<const T*>(p.state);
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / pairs;
    const int col = 2 * (int)(i - t * pairs);
    const uint8_t* row = reinterpret_cast<const uint8_t*>(p.src) + t * p.ld * 4;
    const float2 v = take2<T, true>(row, col);             // raw_n is a multiple of 8
    put2(reinterpret_cast<T*>(p.raw) + t * p.raw_ld, col, v.x, v.y);
    const int c = col - p.col;
    if (c < 0 || c >= p.C) continue;
    const bool two = c + 1 < p.C;
    const int slot = p.sslot[t];
    const bool hist = slot >= 0 && p.ctx[t] > 1;
    const float* wl = p.w + (long long)(p.taps - 1) * p.w_ld + c;
    float a0 = p.b[c] + wl[0] * v.x, a1 = two ? p.b[c + 1] + wl[1] * v.y : 0.f;
    if (hist)
      for (int k = 0; k < p.taps - 1; ++k) {
        const T* r = state + ((long long)slot * (p.taps - 1) + k) * p.C + c;
        a0 += p.w[(long long)k * p.w_ld + c] * Cvt<T>::to_f(r[0]);
        if (two) a1 += p.w[(long long)k * p.w_ld + c + 1] * Cvt<T>::to_f(r[1]);
      }
    T* o = reinterpret_cast<T*>(p.out) + t * p.o_ld + c;
    o[0] = Cvt<T>::from_f(silu_f(a0));
    if (two) o[1] = Cvt<T>::from_f(silu_f(a1));
  }
}

inline int grid_for(long long total, int block) {
  long long g = (total + block - 1) / block;
  const long long cap = (long long)dlti_num_sms() * 16;
  return (int)(g < 1 ? 1 : (g > cap ? cap : g));
}

template <typename T, bool ACC>
int post_norm_add_t(const void* y, long long y_ld, float* x, const float* w, void* xa, long long xa_ld, long long rows, int d,
                    float eps, int one, cudaStream_t st) {
  const int pairs = (d + 2 * PN_THREADS - 1) / (2 * PN_THREADS);
#define PN_CASE(P)                                                                                                      \
  if (pairs <= P) {                                                                                                     \
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, post_norm_add_kernel<T, ACC, P>, dim3((unsigned)rows), dim3(PN_THREADS), 0, st, y, \
                                    y_ld, x, w, (T*)xa, xa_ld, d, eps, one ? 1.f : 0.f));                               \
    dlti_count_launch();                                                                                                \
    return 0;                                                                                                           \
  }
  PN_CASE(1) PN_CASE(2) PN_CASE(4) PN_CASE(8) PN_CASE(16)
#undef PN_CASE
  dlti_set_error("post_norm_add: rows of up to 8192 elements");
  return DLTI_ERR_TOO_LARGE;
}

}  // namespace

#define DISPATCH_T(dtype, CALL)                                      \
  do {                                                               \
    if ((dtype) == DLTI_BF16) { using T = __nv_bfloat16; CALL; }     \
    else if ((dtype) == DLTI_FP32) { using T = float; CALL; }        \
    else return DLTI_ERR_UNSUPPORTED;                                \
  } while (0)

DLTI_API int dlti_embed_rows(const long long* ids, const void* table, float* x, void* xa, long long xa_ld, long long tokens,
                             int d, long long vocab, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  const int g = grid_for(tokens * d, 256);
  DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, embed_rows_kernel<T>, dim3(g), dim3(256), 0, st, ids, (const T*)table, x,
                                                    (T*)xa, xa_ld, tokens, d, vocab)));
  dlti_count_launch();
  return 0;
}

// the decode GEMM's accumulator [rows, cols] as an fp32 result (cols a multiple of 4); zero on return
DLTI_API int dlti_take_rows(float* acc, float* out, long long rows, int cols, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (cols % 4) return DLTI_ERR_BAD_ARG;
  const long long vec = rows * (cols / 4);
  DLTI_CUDA_CHECK(dlti_launch_pdl(rows, take_rows_kernel, dim3(grid_for(vec, 256)), dim3(256), 0, st, acc, out, vec));
  dlti_count_launch();
  return 0;
}

// acc: y is the fp32 accumulator of the decode GEMM (zero on return)
DLTI_API int dlti_post_norm_add(const void* y, long long y_ld, float* x, const float* w, void* xa, long long xa_ld, long long rows,
                                int d, float eps, int one_plus, int acc, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (y_ld % 2) return DLTI_ERR_BAD_ARG;
  if (acc) DISPATCH_T(dtype, return (post_norm_add_t<T, true>(y, y_ld, x, w, xa, xa_ld, rows, d, eps, one_plus, st)));
  DISPATCH_T(dtype, return (post_norm_add_t<T, false>(y, y_ld, x, w, xa, xa_ld, rows, d, eps, one_plus, st)));
}

DLTI_API int dlti_rms_rows(const float* x, const long long* idx, const float* w, void* out, long long out_ld, long long rows, int d,
                           float eps, int one_plus, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, rms_rows_kernel<T>, dim3((unsigned)rows), dim3(PN_THREADS), 0, st, x, idx, w,
                                                    (T*)out, out_ld, d, eps, one_plus ? 1.f : 0.f)));
  dlti_count_launch();
  return 0;
}

DLTI_API int dlti_relu2(const void* u, long long u_ld, void* h, long long h_ld, long long rows, int ff, int acc, int dtype,
                        cudaStream_t st) {
  if (rows <= 0) return 0;
  if (u_ld % 2 || h_ld % 2) return DLTI_ERR_BAD_ARG;
  if (!acc && dtype == DLTI_BF16 && ff % 8 == 0 && u_ld % 8 == 0 && h_ld % 8 == 0 &&
      ((reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(h)) & 15) == 0) {
    relu2_vec_kernel<__nv_bfloat16><<<grid_for(rows * (ff / 8), 256), 256, 0, st>>>((const __nv_bfloat16*)u, u_ld, (__nv_bfloat16*)h,
                                                                                    h_ld, rows, ff);
    dlti_count_launch();
    return (int)cudaGetLastError();
  }
  const int g = grid_for(rows * ((ff + 1) / 2), 256);
  if (acc)
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, relu2_kernel<T, true>, dim3(g), dim3(256), 0, st, u, u_ld, (T*)h, h_ld, rows, ff)));
  else
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, relu2_kernel<T, false>, dim3(g), dim3(256), 0, st, u, u_ld, (T*)h, h_ld, rows, ff)));
  dlti_count_launch();
  return 0;
}

DLTI_API int dlti_gated_norm(const void* y, long long y_ld, const void* gate, long long g_ld, const float* w, void* out, long long o_ld,
                             long long rows, int n, int groups, float eps, int gate_first, int acc, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (groups < 1 || n % groups) return DLTI_ERR_BAD_ARG;
  const size_t smem = (size_t)n * 4;
  if (smem > 48 * 1024) { dlti_set_error("gated_norm: rows of up to 12288 elements"); return DLTI_ERR_TOO_LARGE; }
#define GN_CASE(GF, AC)                                                                                                          \
  DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, gated_norm_kernel<T, GF, AC>, dim3((unsigned)rows), dim3(256), smem, st, \
                                                    (const T*)y, y_ld, gate, g_ld, w, (T*)out, o_ld, n, groups, eps)))
  if (gate_first && acc) GN_CASE(true, true);
  else if (gate_first) GN_CASE(true, false);
  else if (acc) GN_CASE(false, true);
  else GN_CASE(false, false);
#undef GN_CASE
  dlti_count_launch();
  return 0;
}

DLTI_API int dlti_qk_norm_rope_cache(const void* proj, long long ld, int oq, int ok, int ov, int og, const float* qn, const float* kn,
                                     float eps, const int* pos, const float* cos_t, const float* sin_t, int rot, int interleaved,
                                     const long long* slots, void* kc, void* vc, int kd, int vd, void* q, long long q_ld, int q_hd,
                                     void* kp, void* vp, float* gate, long long tokens, int H, int G, int dim, int vdim, int acc,
                                     int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (rot % 2 || rot > dim || ld % 2) return DLTI_ERR_BAD_ARG;
  if (rot / 2 + (dim - rot + 1) / 2 > 32 * QKV_MAXP) { dlti_set_error("qk_norm_rope_cache: heads of up to 512 dimensions"); return DLTI_ERR_TOO_LARGE; }
  QkvParams p{proj, ld, oq, ok, ov, og, qn, kn, eps, pos, cos_t, sin_t, rot, interleaved, slots, kc, vc, kd, vd,
              q, q_ld, q_hd, kp, vp, gate, tokens, H, G, dim, vdim};
  const int jobs = H + ((ok >= 0 || kp) ? 2 * G : 0) + (og >= 0 ? 1 : 0);
  const int g = grid_for(tokens * jobs * 32, 256);
  if (acc) DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, qk_norm_rope_cache_kernel<T, true>, dim3(g), dim3(256), 0, st, p)));
  else DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, qk_norm_rope_cache_kernel<T, false>, dim3(g), dim3(256), 0, st, p)));
  dlti_count_launch();
  return 0;
}

DLTI_API int dlti_short_conv(const void* src, long long ld, int col, int C, int taps, const float* w, const float* b, int w_ld,
                             const void* state, const int* sslot, const int* rseq, const int* ctx, const int* cu, int nd, void* out,
                             long long o_ld, void* raw, long long raw_ld, int raw_n, long long rows, int acc, int dtype,
                             cudaStream_t st) {
  if (rows <= 0) return 0;
  if (taps < 1 || C < 1) return DLTI_ERR_BAD_ARG;
  ConvParams p{src, ld, col, C, taps, w, b, w_ld, state, sslot, rseq, ctx, cu, nd, out, o_ld, raw, raw_ld, raw_n, rows};
  if (acc) {
    if (nd != rows || !raw || raw_n % 2) return DLTI_ERR_BAD_ARG;
    const int g = grid_for(rows * (raw_n / 2), 256);
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, short_conv_acc_kernel<T>, dim3(g), dim3(256), 0, st, p)));
  } else {
    const int g = grid_for(rows * ((C + 1) / 2), 256);
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, short_conv_kernel<T>, dim3(g), dim3(256), 0, st, p)));
  }
  dlti_count_launch();
  return 0;
}

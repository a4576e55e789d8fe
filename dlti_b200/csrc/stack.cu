// Row-wise kernels of the layer-stack models (models/stack.py): fp32 residual stream, norms on the sublayer outputs,
// per-head query/key norm + rotary + paged-cache write, squared relu, gated norms, short causal convolutions.
//
// Residual, norms, gates and rotations are fp32 for either activation type; see rows.cuh for the two forms of a projection.
#include "rows.cuh"

namespace {

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

// out = scale * acc (fp32), with cap > 0: cap * tanh(scale * acc / cap); clear: acc = 0 (otherwise out may be acc)
__global__ void take_rows_kernel(float* acc, float* out, float scale, float cap, int clear, long long vec) {
  griddep_wait();
  griddep_launch();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < vec; i += (long long)gridDim.x * blockDim.x) {
    float4 v = reinterpret_cast<float4*>(acc)[i];
    if (clear) reinterpret_cast<float4*>(acc)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    v = make_float4(scale * v.x, scale * v.y, scale * v.z, scale * v.w);
    if (cap > 0.f) v = make_float4(cap * tanhf(v.x / cap), cap * tanhf(v.y / cap), cap * tanhf(v.z / cap), cap * tanhf(v.w / cap));
    reinterpret_cast<float4*>(out)[i] = v;
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

// the same in 16-byte pieces, every load issued before the reduction: 16-bit T, d and pitches multiples of 8
template <typename T, bool ACC, int VPT>
__global__ void __launch_bounds__(128) post_norm_add_vec_kernel(const void* __restrict__ y, long long y_ld, float* __restrict__ x,
                                                               const float* __restrict__ w, T* __restrict__ xa, long long xa_ld,
                                                               int d, float eps, float one) {
  __shared__ float red[32];
  const int vec = d >> 3;
  float wv[VPT][8];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {                   // weights never change: they may come before the wait
    const int v = threadIdx.x + i * 128;
    if (v < vec) ld8(w + v * 8, wv[i]);
  }
  griddep_wait();
  griddep_launch();
  const long long row = blockIdx.x;
  const void* yr = reinterpret_cast<const uint8_t*>(y) + row * y_ld * (ACC ? 4 : sizeof(T));
  float* xr = x + row * d;
  float yv[VPT][8], xv[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * 128;
    if (v < vec) {
      take_n<T, ACC, 8>(yr, v * 8, yv[i]);
      ld8(xr + v * 8, xv[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (threadIdx.x + i * 128 < vec)
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += yv[i][j] * yv[i][j];
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)d + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * 128;
    if (v < vec) {
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[i][j] += yv[i][j] * r * (one + wv[i][j]);
      st8(xr + v * 8, xv[i]);
      if (xa) put_n(xa + row * xa_ld + v * 8, xv[i]);
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
template <typename T, bool ACC>
__global__ void relu2_vec_kernel(const void* __restrict__ u, long long u_ld, T* __restrict__ h, long long h_ld, long long rows, int ff) {
  griddep_wait();
  griddep_launch();
  const int vec = ff >> 3;
  const long long total = rows * vec;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / vec;
    const int c = 8 * (int)(i - t * vec);
    float f[8];
    take_n<T, ACC, 8>(reinterpret_cast<const uint8_t*>(u) + t * u_ld * (ACC ? 4 : sizeof(T)), c, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      f[j] = fmaxf(f[j], 0.f);
      f[j] *= f[j];
    }
    put_n(h + t * h_ld + c, f);
  }
}

// Norm of a mixer output in `groups` equal parts with a multiplicative gate.
//   GATE_SILU_FIRST:  out = norm(y * silu(g)) * w          (Mamba-2)
//   GATE_SIGMOID:     out = norm(y) * w * sigmoid(g)       (lightning attention, mLSTM)
//   GATE_SILU:        out = norm(y) * w * silu(g)          (delta rule)
// One CTA per row, one warp per group in turn; a group is passed twice (second time from L1).
enum Gate : int { GATE_SIGMOID = 0, GATE_SILU_FIRST = 1, GATE_SILU = 2 };
template <typename T, int GATE, bool ACC>
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
    row_s[c] = GATE == GATE_SILU_FIRST ? Cvt<T>::to_f(yr[c]) * silu_f(g) : GATE == GATE_SILU ? silu_f(g) : sigmoid_f(g);
  }
  __syncthreads();
  if (groups == 1) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float v = GATE == GATE_SILU_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]);
      ss += v * v;
    }
    ss = block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / (float)n + eps);
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float v = (GATE == GATE_SILU_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]) * row_s[c]) * r * w[c];
      out[t * o_ld + c] = Cvt<T>::from_f(v);
    }
    return;
  }
  for (int g = threadIdx.x >> 5; g < groups; g += blockDim.x >> 5) {
    float ss = 0.f;
    for (int c = g * gs + (threadIdx.x & 31); c < (g + 1) * gs; c += 32) {
      const float v = GATE == GATE_SILU_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]);
      ss += v * v;
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)gs + eps);
    for (int c = g * gs + (threadIdx.x & 31); c < (g + 1) * gs; c += 32) {
      const float v = (GATE == GATE_SILU_FIRST ? row_s[c] : Cvt<T>::to_f(yr[c]) * row_s[c]) * r * w[c];
      out[t * o_ld + c] = Cvt<T>::from_f(v);
    }
  }
}

// the same in 16-byte pieces for 16-bit T and groups of whole pieces: one CTA per (row, group), everything in registers
template <typename T, int GATE, bool ACC, int VPT>
__global__ void __launch_bounds__(512) gated_norm_vec_kernel(const T* __restrict__ y, long long y_ld, const void* __restrict__ gate,
                                                             long long g_ld, const float* __restrict__ w, T* __restrict__ out,
                                                             long long o_ld, int gs, float eps) {
  __shared__ float red[32];
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  const int c0 = blockIdx.y * gs, vec = gs >> 3;
  const T* yr = y + t * y_ld;
  const void* gr = reinterpret_cast<const uint8_t*>(gate) + t * g_ld * (ACC ? 4 : sizeof(T));
  float v[VPT][8], g[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int p = threadIdx.x + i * blockDim.x;
    if (p < vec) {
      take_n<T, false, 8>(yr, c0 + p * 8, v[i]);
      take_n<T, ACC, 8>(gr, c0 + p * 8, g[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (threadIdx.x + i * blockDim.x < vec)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float e = fast_sigmoid(g[i][j]);
        if (GATE == GATE_SILU_FIRST) v[i][j] *= g[i][j] * e;
        else g[i][j] = GATE == GATE_SILU ? g[i][j] * e : e;
        ss += v[i][j] * v[i][j];
      }
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)gs + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int p = threadIdx.x + i * blockDim.x;
    if (p < vec) {
      float wv[8];
      ld8(w + c0 + p * 8, wv);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= r * wv[j] * (GATE == GATE_SILU_FIRST ? 1.f : g[i][j]);
      put_n(out + t * o_ld + c0 + p * 8, v[i]);
    }
  }
}

// many small groups: LPG lanes per group (VPT > 1: a warp)
template <typename T, int GATE, bool ACC, int VPT, int LPG>
__global__ void __launch_bounds__(256) gated_norm_warp_kernel(const T* __restrict__ y, long long y_ld, const void* __restrict__ gate,
                                                              long long g_ld, const float* __restrict__ w, T* __restrict__ out,
                                                              long long o_ld, int gs, int groups, long long total, float eps) {
  griddep_wait();
  griddep_launch();
  const long long x0 = ((long long)blockIdx.x * 256 + threadIdx.x) / LPG, x = min(x0, total - 1);       // whole warps take part in the sums
  const long long t = x / groups;
  const int c0 = (int)(x - t * groups) * gs, vec = x0 < total ? gs >> 3 : 0, lane = threadIdx.x % LPG;
  const T* yr = y + t * y_ld;
  const void* gr = reinterpret_cast<const uint8_t*>(gate) + t * g_ld * (ACC ? 4 : sizeof(T));
  float v[VPT][8], g[VPT][8], ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (lane + LPG * i < vec) {
      take_n<T, false, 8>(yr, c0 + (lane + LPG * i) * 8, v[i]);
      take_n<T, ACC, 8>(gr, c0 + (lane + LPG * i) * 8, g[i]);
    }
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (lane + LPG * i < vec)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float e = fast_sigmoid(g[i][j]);
        if (GATE == GATE_SILU_FIRST) v[i][j] *= g[i][j] * e;
        else g[i][j] = GATE == GATE_SILU ? g[i][j] * e : e;
        ss += v[i][j] * v[i][j];
      }
#pragma unroll
  for (int o = LPG / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = 1.f / sqrtf(ss / (float)gs + eps);
  if (x0 >= total) return;
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (lane + LPG * i < vec) {
      float wv[8];
      ld8(w + c0 + (lane + LPG * i) * 8, wv);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= r * wv[j] * (GATE == GATE_SILU_FIRST ? 1.f : g[i][j]);
      put_n(out + t * o_ld + c0 + (lane + LPG * i) * 8, v[i]);
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
  const int* dst; int nd;                                  // packed: row of token t >= nd is nd + dst[t - nd] (null: t)
  float* gate;                                             // [tokens, H]
  long long tokens; int H, G, dim, vdim;
};
__device__ __forceinline__ long long q_row(const QkvParams& p, long long t) {
  return (p.dst && t >= p.nd) ? p.nd + (long long)p.dst[t - p.nd] : t;
}
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
      T* pk = p.vp ? reinterpret_cast<T*>(p.vp) + q_row(p, t) * p.q_ld + (long long)g * p.q_hd : nullptr;
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
    T* out = is_q ? reinterpret_cast<T*>(p.q) + q_row(p, t) * p.q_ld + (long long)head * p.q_hd
                  : (p.kp ? reinterpret_cast<T*>(p.kp) + q_row(p, t) * p.q_ld + (long long)head * p.q_hd : nullptr);
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

// The same for heads of 8 * LPH (64, 128, 256) elements, interleaved pairs and 16-byte aligned sections: LPH lanes share a
// head (8 consecutive elements each, so a lane's rotation factors are the same for every head), a warp takes 32 / LPH heads
// of one token at a time and JPW such groups with all their loads in flight.
template <typename T, bool ACC, int LPH, int JPW>
__global__ void __launch_bounds__(128) qk_norm_rope_cache_vec_kernel(const QkvParams p, int jobs, int kvjobs) {
  constexpr int HPW = 32 / LPH, HD = 8 * LPH;
  griddep_wait();
  griddep_launch();
  const int lane = threadIdx.x & 31, sub = lane % LPH, e0 = sub * 8, half = p.rot >> 1;
  const long long t = blockIdx.x;
  const int job0 = (blockIdx.y * 4 + (threadIdx.x >> 5)) * (HPW * JPW);
  if (job0 >= jobs) return;
  const uint8_t* row = reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * (ACC ? 4 : sizeof(T));
  const long long slot = p.slots[t];
  const int ps = p.pos[t];
  const long long to = q_row(p, t);
  const bool own = p.ok >= 0;
  float v[JPW][8];
#pragma unroll
  for (int i = 0; i < JPW; ++i) {
    const int job = job0 + i * HPW + lane / LPH;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[i][j] = 0.f;
    if (job < p.H) {
      take_n<T, ACC, 8>(row, p.oq + job * HD + e0, v[i]);
    } else if (job < p.H + kvjobs) {
      const bool is_k = job < p.H + p.G;
      const int g = is_k ? job - p.H : job - p.H - p.G;      // G keys, then G values
      if (own) take_n<T, ACC, 8>(row, (is_k ? p.ok : p.ov) + g * HD + e0, v[i]);
      else if (slot >= 0)
        take_n<T, false, 8>(reinterpret_cast<const T*>(is_k ? p.kc : p.vc) + (slot * p.G + g) * (is_k ? p.kd : p.vd), e0, v[i]);
    }
  }
  float cs[4], sn[4], wq[8], wk[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) wq[j] = wk[j] = 1.f;
  if (p.qn) ld8(p.qn + e0, wq);
  if (p.kn) ld8(p.kn + e0, wk);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int pr = e0 / 2 + j;
    cs[j] = pr < half ? p.cos_t[(long long)ps * half + pr] : 1.f;
    sn[j] = pr < half ? p.sin_t[(long long)ps * half + pr] : 0.f;
  }
#pragma unroll
  for (int i = 0; i < JPW; ++i) {
    const int job = job0 + i * HPW + lane / LPH;
    const bool is_q = job < p.H, is_v = job >= p.H + p.G;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[i][j] * v[i][j];
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);     // whole warp, also past the last job
    if (job >= jobs) continue;
    if (job >= p.H + kvjobs) {
      for (int h = sub; h < p.H; h += LPH) p.gate[t * p.H + h] = sigmoid_f(take<T, ACC>(row, p.og + h));
      continue;
    }
    if (is_q || (own && !is_v)) {
      const float r = (is_q ? p.qn : p.kn) ? rsqrtf(ss * (1.f / HD) + p.eps) : 1.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float a = v[i][2 * j] * r * (is_q ? wq[2 * j] : wk[2 * j]), b = v[i][2 * j + 1] * r * (is_q ? wq[2 * j + 1] : wk[2 * j + 1]);
        v[i][2 * j] = a * cs[j] - b * sn[j];
        v[i][2 * j + 1] = b * cs[j] + a * sn[j];
      }
    }
    if (is_q) {
      put_n(reinterpret_cast<T*>(p.q) + to * p.q_ld + job * p.q_hd + e0, v[i]);
    } else {
      const int g = is_v ? job - p.H - p.G : job - p.H;
      void* pk = is_v ? p.vp : p.kp;
      if (pk) put_n(reinterpret_cast<T*>(pk) + to * p.q_ld + g * p.q_hd + e0, v[i]);
      if (own && slot >= 0) put_n(reinterpret_cast<T*>(is_v ? p.vc : p.kc) + (slot * p.G + g) * (is_v ? p.vd : p.kd) + e0, v[i]);
    }
  }
}

// Whole projection rows: bias, norm of q and of k over all their heads, values mixed with those of an earlier layer, cache
// write of k and v. One CTA per token; the row waits in shared memory for its norms. W: elements per piece (8: 16-bit T, head
// sizes and pitches multiples of 8).
struct QkvRowParams {
  const void* proj; long long ld; int oq, ok, ov;
  const float *bias, *qn, *kn; float eps;                  // bias: laid out as the projection; any of them may be null
  const void* first; long long f_ld; const float* share;   // values to mix in [tokens, G * vdim] and their share (null: none)
  void* own; long long own_ld;                             // copy of the values before mixing (null: none)
  const long long* slots; void *kc, *vc; int kd, vd;
  void* q; long long q_ld; int q_hd;
  void *kp, *vp; const int* dst; int nd;                   // packed keys / values, as in QkvParams
  int H, G, dim, vdim;
};
template <typename T, bool ACC, int W>
__device__ __forceinline__ void row_piece(const void* row, const float* bias, int c, float (&f)[W]) {
  if constexpr (W == 1) f[0] = take<T, ACC>(row, c);
  else take_n<T, ACC, W>(row, c, f);
  if (bias) {
#pragma unroll
    for (int j = 0; j < W; ++j) f[j] += bias[c + j];
  }
}
template <typename T, int W>
__device__ __forceinline__ void put_piece(T* p, const float (&f)[W]) {
  if constexpr (W == 1) *p = Cvt<T>::from_f(f[0]);
  else put_n(p, f);
}
template <typename T, bool ACC, int W>
__global__ void __launch_bounds__(256) qkv_rows_kernel(const QkvRowParams p) {
  __shared__ float red[32];
  extern __shared__ __align__(16) float row_q[];           // q, then k
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  const uint8_t* row = reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * (ACC ? 4 : sizeof(T));
  const long long slot = p.slots[t];
  const long long to = (p.dst && t >= p.nd) ? p.nd + (long long)p.dst[t - p.nd] : t;
  const int nq = p.H * p.dim, nk = p.G * p.dim, nv = p.G * p.vdim;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x * W; i < nq + nk; i += blockDim.x * W) {
    float f[W];
    row_piece<T, ACC, W>(row, p.bias, i < nq ? p.oq + i : p.ok + i - nq, f);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < W; ++j) {
      ss += f[j] * f[j];
      row_q[i + j] = f[j];
    }
    if (i < nq) sq += ss;
    else sk += ss;
  }
  const float share = p.first ? p.share[0] : 0.f;
  for (int i = threadIdx.x * W; i < nv; i += blockDim.x * W) {
    float f[W];
    row_piece<T, ACC, W>(row, p.bias, p.ov + i, f);
    if (p.own) put_piece<T, W>(reinterpret_cast<T*>(p.own) + t * p.own_ld + i, f);
    if (p.first) {
      float e[W];
      row_piece<T, false, W>(reinterpret_cast<const T*>(p.first) + t * p.f_ld, nullptr, i, e);
#pragma unroll
      for (int j = 0; j < W; ++j) f[j] += share * (e[j] - f[j]);
    }
    const int g = i / p.vdim, c = i - g * p.vdim;
    if (p.vp) put_piece<T, W>(reinterpret_cast<T*>(p.vp) + to * p.q_ld + (long long)g * p.q_hd + c, f);
    if (slot >= 0) put_piece<T, W>(reinterpret_cast<T*>(p.vc) + (slot * p.G + g) * p.vd + c, f);
  }
  float rq = 1.f, rk = 1.f;
  if (p.qn) {
    rq = 1.f / sqrtf(block_sum(sq, red) / (float)nq + p.eps);
    rk = 1.f / sqrtf(block_sum(sk, red) / (float)nk + p.eps);
  }
  for (int i = threadIdx.x * W; i < nq + nk; i += blockDim.x * W) {      // a thread's own pieces: no barrier needed
    const bool is_q = i < nq;
    const int x = is_q ? i : i - nq, h = x / p.dim, c = x - h * p.dim;
    float f[W];
#pragma unroll
    for (int j = 0; j < W; ++j) {
      f[j] = row_q[i + j];
      if (p.qn) f[j] *= (is_q ? rq : rk) * (is_q ? p.qn : p.kn)[x + j];
    }
    if (is_q) {
      put_piece<T, W>(reinterpret_cast<T*>(p.q) + to * p.q_ld + (long long)h * p.q_hd + c, f);
    } else {
      if (p.kp) put_piece<T, W>(reinterpret_cast<T*>(p.kp) + to * p.q_ld + (long long)h * p.q_hd + c, f);
      if (slot >= 0) put_piece<T, W>(reinterpret_cast<T*>(p.kc) + (slot * p.G + h) * p.kd + c, f);
    }
  }
}

// the same with the row in registers: 16-bit T, VPT pieces of 8 a thread, every load issued before the sums
template <typename T, bool ACC, int VPT, int THREADS>
__global__ void __launch_bounds__(THREADS) qkv_rows_vec_kernel(const QkvRowParams p) {
  __shared__ float2 red[THREADS / 32];
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  const uint8_t* row = reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * (ACC ? 4 : sizeof(T));
  const long long slot = p.slots[t];
  const long long to = (p.dst && t >= p.nd) ? p.nd + (long long)p.dst[t - p.nd] : t;
  const int nq = p.H * p.dim, nk = p.G * p.dim, nv = p.G * p.vdim;
  float f[VPT][8], sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int x = (threadIdx.x + i * THREADS) * 8;
    if (x < nq + nk + nv) take_n<T, ACC, 8>(row, x < nq ? p.oq + x : x < nq + nk ? p.ok + x - nq : p.ov + x - nq - nk, f[i]);
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int x = (threadIdx.x + i * THREADS) * 8;
    if (x >= nq + nk + nv) continue;
    if (p.bias) {
      float b[8];
      ld8(p.bias + (x < nq ? p.oq + x : x < nq + nk ? p.ok + x - nq : p.ov + x - nq - nk), b);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[i][j] += b[j];
    }
    if (x < nq + nk) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += f[i][j] * f[i][j];
      if (x < nq) sq += ss;
      else sk += ss;
    }
  }
  float rq = 1.f, rk = 1.f;
  if (p.qn) {
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(sq, sk);
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) {
      sq += red[w].x;
      sk += red[w].y;
    }
    rq = rsqrtf(sq / (float)nq + p.eps);
    rk = rsqrtf(sk / (float)nk + p.eps);
  }
  const float share = p.first ? p.share[0] : 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int x = (threadIdx.x + i * THREADS) * 8;
    if (x >= nq + nk + nv) continue;
    const bool is_q = x < nq, is_v = x >= nq + nk;
    const int y = is_q ? x : is_v ? x - nq - nk : x - nq, hd = is_v ? p.vdim : p.dim, h = y / hd, c = y - h * hd;
    if (is_v) {
      if (p.own) put_n(reinterpret_cast<T*>(p.own) + t * p.own_ld + y, f[i]);
      if (p.first) {
        float e[8];
        take_n<T, false, 8>(reinterpret_cast<const T*>(p.first) + t * p.f_ld, y, e);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[i][j] += share * (e[j] - f[i][j]);
      }
    } else if (p.qn) {
      float w[8];
      ld8((is_q ? p.qn : p.kn) + y, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[i][j] *= (is_q ? rq : rk) * w[j];
    }
    if (is_q) {
      put_n(reinterpret_cast<T*>(p.q) + to * p.q_ld + (long long)h * p.q_hd + c, f[i]);
    } else {
      void* pk = is_v ? p.vp : p.kp;
      if (pk) put_n(reinterpret_cast<T*>(pk) + to * p.q_ld + (long long)h * p.q_hd + c, f[i]);
      if (slot >= 0) put_n(reinterpret_cast<T*>(is_v ? p.vc : p.kc) + (slot * p.G + h) * (is_v ? p.vd : p.kd) + c, f[i]);
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
  float* tail; long long tail_ld; int tail0;               // accumulator columns from tail0 on go here unrounded (null: nowhere)
};
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
// The same, 8 channels x CONV_ROWS rows per thread with the window in registers (16-bit T, C and pitches multiples of 8,
// TAPS fixed). Row blocks that touch the start of a sequence read rows or state tap by tap.
constexpr int CONV_ROWS = 8;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) short_conv_vec_kernel(const ConvParams p) {
  griddep_wait();
  griddep_launch();
  const int vec = p.C >> 3, cv = blockIdx.y * 128 + threadIdx.x;
  if (cv >= vec) return;
  const int c = cv * 8;
  const long long t0 = (long long)blockIdx.x * CONV_ROWS;
  const int nr = (int)min((long long)CONV_ROWS, p.rows - t0);
  const T* src = reinterpret_cast<const T*>(p.src) + p.col + c;
  const T* state = reinterpret_cast<const T*>(p.state) + c;
  float w[TAPS][8], b[8];
#pragma unroll
  for (int k = 0; k < TAPS; ++k) ld8(p.w + (long long)k * p.w_ld + c, w[k]);
  ld8(p.b + c, b);
  T* out = reinterpret_cast<T*>(p.out) + c;
  const int s0 = p.rseq[t0];
  long long row0;
  int n, start;
  seq_rows(p.cu, p.ctx, p.nd, s0, row0, n, start);
  auto emit = [&](long long t, const float (&a)[8]) {
    float f[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = a[j] * fast_sigmoid(a[j]);
    put_n(out + t * p.o_ld, f);
  };
  if (t0 - row0 >= TAPS - 1 && t0 + nr <= row0 + n) {            // all inputs are rows of this step
    uint4 x[TAPS - 1 + CONV_ROWS];                               // still packed: all loads in flight at half the registers
    const T* sp = src + (t0 - (TAPS - 1)) * p.ld;
#pragma unroll
    for (int i = 0; i < TAPS - 1 + CONV_ROWS; ++i)
      if (i < TAPS - 1 + nr) x[i] = *reinterpret_cast<const uint4*>(sp + i * p.ld);
#pragma unroll
    for (int r = 0; r < CONV_ROWS; ++r)
      if (r < nr) {
        float a[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] = b[j];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) {
          const uint32_t u[4] = {x[r + k].x, x[r + k].y, x[r + k].z, x[r + k].w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float2 f = Cvt<T>::unpack2(u[j]);
            a[2 * j] += w[k][2 * j] * f.x;
            a[2 * j + 1] += w[k][2 * j + 1] * f.y;
          }
        }
        emit(t0 + r, a);
      }
    return;
  }
  for (int r = 0; r < nr; ++r) {
    const long long t = t0 + r;
    const int s = p.rseq[t];
    seq_rows(p.cu, p.ctx, p.nd, s, row0, n, start);
    const int local = (int)(t - row0), slot = p.sslot[s];
    float a[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] = b[j];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      const int q = local - (TAPS - 1) + k;
      float x[8];
      if (q >= 0) take_n<T, false, 8>(src + (row0 + q) * p.ld, 0, x);
      else if (start > 0 && slot >= 0) take_n<T, false, 8>(state + ((long long)slot * (TAPS - 1) + q + TAPS - 1) * p.C, 0, x);
      else continue;
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] += w[k][j] * x[j];
    }
    emit(t, a);
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
    if (p.tail && col >= p.tail0) {
      const float2 v = take2<float, true>(row, col);
      *reinterpret_cast<float2*>(p.tail + t * p.tail_ld + col - p.tail0) = v;
      continue;
    }
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

// the same, 8 columns per thread (C, col and every pitch multiples of 8)
template <typename T>
__global__ void __launch_bounds__(128) short_conv_acc_vec_kernel(const ConvParams p) {
  griddep_wait();
  griddep_launch();
  const int col = (blockIdx.y * 128 + threadIdx.x) * 8;
  if (col >= p.raw_n) return;
  const long long t = blockIdx.x;
  float v[8];
  if (p.tail && col >= p.tail0) {
    take_n<float, true, 8>(reinterpret_cast<const uint8_t*>(p.src) + t * p.ld * 4, col, v);
    st8(p.tail + t * p.tail_ld + col - p.tail0, v);
    return;
  }
  take_n<T, true, 8>(reinterpret_cast<const uint8_t*>(p.src) + t * p.ld * 4, col, v);
  put_n(reinterpret_cast<T*>(p.raw) + t * p.raw_ld + col, v);
  const int c = col - p.col;
  if (c < 0 || c >= p.C) return;
  const int slot = p.sslot[t];
  float a[8], w[8];
  ld8(p.b + c, a);
  ld8(p.w + (long long)(p.taps - 1) * p.w_ld + c, w);
#pragma unroll
  for (int j = 0; j < 8; ++j) a[j] += w[j] * v[j];
  if (slot >= 0 && p.ctx[t] > 1) {
    const T* st = reinterpret_cast<const T*>(p.state) + (long long)slot * (p.taps - 1) * p.C + c;
#pragma unroll 3
    for (int k = 0; k < p.taps - 1; ++k) {
      float x[8];
      take_n<T, false, 8>(st + (long long)k * p.C, 0, x);
      ld8(p.w + (long long)k * p.w_ld + c, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] += w[j] * x[j];
    }
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) a[j] *= fast_sigmoid(a[j]);
  put_n(reinterpret_cast<T*>(p.out) + t * p.o_ld + c, a);
}

// Cached keys and values in front of a portion's rows: packed row rows[i] <- zero queries, keys and values of slot slots[i].
// 16-byte pieces; heads are `hd` columns apart in the packed rows and kd / vd in the cache.
__global__ void prefix_rows_kernel(__nv_bfloat16* __restrict__ packed, long long ld, int hd, const int* __restrict__ rows,
                                   const int* __restrict__ slots, const __nv_bfloat16* __restrict__ kc,
                                   const __nv_bfloat16* __restrict__ vc, int kd, int vd, int H, int G, long long total) {
  const int pieces = (H + 2 * G) * (hd / 8);
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / pieces;
    const int x = (int)(i - r * pieces), head = x / (hd / 8), c = x % (hd / 8) * 8;
    int4 v = make_int4(0, 0, 0, 0);
    if (head >= H) {
      const bool is_k = head < H + G;
      const int g = is_k ? head - H : head - H - G, w = is_k ? kd : vd;
      if (c < w) v = *reinterpret_cast<const int4*>((is_k ? kc : vc) + ((long long)slots[r] * G + g) * w + c);
    }
    *reinterpret_cast<int4*>(packed + (long long)rows[r] * ld + head * hd + c) = v;
  }
}

template <typename T, bool ACC>
int post_norm_add_t(const void* y, long long y_ld, float* x, const float* w, void* xa, long long xa_ld, long long rows, int d,
                    float eps, int one, cudaStream_t st) {
  if constexpr (sizeof(T) == 2) {
    if (d % 8 == 0 && d <= 8192 && y_ld % 8 == 0 && (!xa || xa_ld % 8 == 0) &&
        ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(xa)) & 15) == 0) {
      const int vpt = (d / 8 + 127) / 128;
      auto kern = vpt <= 1 ? post_norm_add_vec_kernel<T, ACC, 1> : vpt <= 2 ? post_norm_add_vec_kernel<T, ACC, 2>
                  : vpt <= 4 ? post_norm_add_vec_kernel<T, ACC, 4> : post_norm_add_vec_kernel<T, ACC, 8>;
      DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kern, dim3((unsigned)rows), dim3(128), 0, st, y, y_ld, x, w, (T*)xa, xa_ld, d, eps,
                                      one ? 1.f : 0.f));
      dlti_count_launch();
      return 0;
    }
  }
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

template <int GATE>
int gated_norm_mode(const void* y, long long y_ld, const void* gate, long long g_ld, const float* w, void* out, long long o_ld, long long rows,
                    int n, int groups, float eps, int acc, int dtype, cudaStream_t st) {
  const int gs = n / groups;
  if (dtype == DLTI_BF16 && gs % 8 == 0 && gs <= 8 * 512 * 4 && y_ld % 8 == 0 && g_ld % 8 == 0 && o_ld % 8 == 0 && groups <= 65535 &&
      ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15) == 0) {
    using B = __nv_bfloat16;
    if (groups > 1 && gs <= 512) {
#define GNW(AC) (gs <= 64 ? gated_norm_warp_kernel<B, GATE, AC, 1, 8> : gs <= 128 ? gated_norm_warp_kernel<B, GATE, AC, 1, 16> \
                 : gs <= 256 ? gated_norm_warp_kernel<B, GATE, AC, 1, 32> : gated_norm_warp_kernel<B, GATE, AC, 2, 32>)
      auto kern = acc ? GNW(true) : GNW(false);
#undef GNW
      const long long total = rows * groups, per = 256 / (gs <= 64 ? 8 : gs <= 128 ? 16 : 32);
      DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kern, dim3((unsigned)((total + per - 1) / per)), dim3(256), 0, st, (const B*)y, y_ld, gate, g_ld, w, (B*)out,
                                      o_ld, gs, groups, total, eps));
      dlti_count_launch();
      return 0;
    }
    const int vec = gs / 8, threads = vec <= 64 ? 64 : (vec <= 128 ? 128 : (vec <= 512 ? 256 : 512)), vpt = (vec + threads - 1) / threads;
#define GNV(AC) (vpt <= 1 ? gated_norm_vec_kernel<B, GATE, AC, 1> : vpt <= 2 ? gated_norm_vec_kernel<B, GATE, AC, 2> : gated_norm_vec_kernel<B, GATE, AC, 4>)
    auto kern = acc ? GNV(true) : GNV(false);
#undef GNV
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kern, dim3((unsigned)rows, groups), dim3(threads), 0, st, (const B*)y, y_ld, gate, g_ld, w, (B*)out,
                                    o_ld, gs, eps));
    dlti_count_launch();
    return 0;
  }
  const size_t smem = (size_t)n * 4;
  if (smem > 48 * 1024) { dlti_set_error("gated_norm: rows of up to 12288 elements"); return DLTI_ERR_TOO_LARGE; }
#define GN_CASE(AC)                                                                                                            \
  DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, gated_norm_kernel<T, GATE, AC>, dim3((unsigned)rows), dim3(256), smem, st, \
                                                    (const T*)y, y_ld, gate, g_ld, w, (T*)out, o_ld, n, groups, eps)))
  if (acc) GN_CASE(true);
  else GN_CASE(false);
#undef GN_CASE
  dlti_count_launch();
  return 0;
}

}  // namespace

DLTI_API int dlti_embed_rows(const long long* ids, const void* table, float* x, void* xa, long long xa_ld, long long tokens,
                             int d, long long vocab, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  const int g = grid_for(tokens * d, 256);
  DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, embed_rows_kernel<T>, dim3(g), dim3(256), 0, st, ids, (const T*)table, x,
                                                    (T*)xa, xa_ld, tokens, d, vocab)));
  dlti_count_launch();
  return 0;
}

// [rows, cols] times scale as an fp32 result (cols a multiple of 4), softly capped with cap > 0. clear: acc is the decode GEMM's
// accumulator, zero on return; otherwise out may be acc.
DLTI_API int dlti_take_rows(float* acc, float* out, float scale, float cap, int clear, long long rows, int cols, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (cols % 4 || cap < 0.f || (clear && acc == out)) return DLTI_ERR_BAD_ARG;
  const long long vec = rows * (cols / 4);
  DLTI_CUDA_CHECK(dlti_launch_pdl(rows, take_rows_kernel, dim3(grid_for(vec, 256)), dim3(256), 0, st, acc, out, scale, cap, clear, vec));
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
  if (dtype == DLTI_BF16 && ff % 8 == 0 && u_ld % 8 == 0 && h_ld % 8 == 0 &&
      ((reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(h)) & 15) == 0) {
    const dim3 g(grid_for(rows * (ff / 8), 256));
    auto kern = acc ? relu2_vec_kernel<__nv_bfloat16, true> : relu2_vec_kernel<__nv_bfloat16, false>;
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kern, g, dim3(256), 0, st, u, u_ld, (__nv_bfloat16*)h, h_ld, rows, ff));
    dlti_count_launch();
    return 0;
  }
  const int g = grid_for(rows * ((ff + 1) / 2), 256);
  if (acc)
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, relu2_kernel<T, true>, dim3(g), dim3(256), 0, st, u, u_ld, (T*)h, h_ld, rows, ff)));
  else
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, relu2_kernel<T, false>, dim3(g), dim3(256), 0, st, u, u_ld, (T*)h, h_ld, rows, ff)));
  dlti_count_launch();
  return 0;
}

// mode: see Gate
DLTI_API int dlti_gated_norm(const void* y, long long y_ld, const void* gate, long long g_ld, const float* w, void* out, long long o_ld,
                             long long rows, int n, int groups, float eps, int mode, int acc, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (groups < 1 || n % groups || mode < 0 || mode > 2) return DLTI_ERR_BAD_ARG;
  if (mode == GATE_SILU_FIRST) return gated_norm_mode<GATE_SILU_FIRST>(y, y_ld, gate, g_ld, w, out, o_ld, rows, n, groups, eps, acc, dtype, st);
  if (mode == GATE_SILU) return gated_norm_mode<GATE_SILU>(y, y_ld, gate, g_ld, w, out, o_ld, rows, n, groups, eps, acc, dtype, st);
  return gated_norm_mode<GATE_SIGMOID>(y, y_ld, gate, g_ld, w, out, o_ld, rows, n, groups, eps, acc, dtype, st);
}

DLTI_API int dlti_qk_norm_rope_cache(const void* proj, long long ld, int oq, int ok, int ov, int og, const float* qn, const float* kn,
                                     float eps, const int* pos, const float* cos_t, const float* sin_t, int rot, int interleaved,
                                     const long long* slots, void* kc, void* vc, int kd, int vd, void* q, long long q_ld, int q_hd,
                                     void* kp, void* vp, const int* dst, int nd, float* gate, long long tokens, int H, int G, int dim, int vdim, int acc,
                                     int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (rot % 2 || rot > dim || ld % 2) return DLTI_ERR_BAD_ARG;
  if (rot / 2 + (dim - rot + 1) / 2 > 32 * QKV_MAXP) { dlti_set_error("qk_norm_rope_cache: heads of up to 512 dimensions"); return DLTI_ERR_TOO_LARGE; }
  QkvParams p{proj, ld, oq, ok, ov, og, qn, kn, eps, pos, cos_t, sin_t, rot, interleaved, slots, kc, vc, kd, vd,
              q, q_ld, q_hd, kp, vp, dst, nd, gate, tokens, H, G, dim, vdim};
  const int kvjobs = (ok >= 0 || kp) ? 2 * G : 0, jobs = H + kvjobs + (og >= 0 ? 1 : 0);
  const bool vec = dtype == DLTI_BF16 && (dim == 64 || dim == 128 || dim == 256) && vdim == dim && (interleaved || rot == 0) && ld % 8 == 0 &&
                   q_ld % 8 == 0 && q_hd % 8 == 0 && kd % 8 == 0 && vd % 8 == 0 && oq % 8 == 0 && (ok < 0 || (ok % 8 == 0 && ov % 8 == 0)) &&
                   tokens < (1ll << 31) &&
                   ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kc) |
                     reinterpret_cast<uintptr_t>(vc) | reinterpret_cast<uintptr_t>(kp) | reinterpret_cast<uintptr_t>(vp) | reinterpret_cast<uintptr_t>(qn) |
                     reinterpret_cast<uintptr_t>(kn)) & 15) == 0;
  if (vec) {
    using B = __nv_bfloat16;
#define QKV_CASE(LPH)                                                                                                            \
  if (dim == 8 * LPH) {                                                                                                          \
    const int per = 4 * (32 / LPH) * (acc ? 1 : 2);                                                                              \
    auto kern = acc ? qk_norm_rope_cache_vec_kernel<B, true, LPH, 1> : qk_norm_rope_cache_vec_kernel<B, false, LPH, 2>;            \
    DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, kern, dim3((unsigned)tokens, (jobs + per - 1) / per), dim3(128), 0, st, p, jobs, kvjobs)); \
  }
    QKV_CASE(8) QKV_CASE(16) QKV_CASE(32)
#undef QKV_CASE
    dlti_count_launch();
    return 0;
  }
  const int g = grid_for(tokens * jobs * 32, 256);
  if (acc) DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, qk_norm_rope_cache_kernel<T, true>, dim3(g), dim3(256), 0, st, p)));
  else DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, qk_norm_rope_cache_kernel<T, false>, dim3(g), dim3(256), 0, st, p)));
  dlti_count_launch();
  return 0;
}

// bias, qn / kn, first / share, own, kp / vp / dst may be null; see QkvRowParams
DLTI_API int dlti_qkv_rows(const void* proj, long long ld, int oq, int ok, int ov, const float* bias, const float* qn, const float* kn, float eps,
                           const void* first, long long f_ld, const float* share, void* own, long long own_ld, const long long* slots, void* kc,
                           void* vc, int kd, int vd, void* q, long long q_ld, int q_hd, void* kp, void* vp, const int* dst, int nd,
                           long long tokens, int H, int G, int dim, int vdim, int acc, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (H % G || dim < 1 || vdim < 1 || (qn == nullptr) != (kn == nullptr) || (first && !share)) return DLTI_ERR_BAD_ARG;
  QkvRowParams p{proj, ld, oq, ok, ov, bias, qn, kn, eps, first, f_ld, share, own, own_ld, slots, kc, vc, kd, vd, q, q_ld, q_hd, kp, vp, dst, nd,
                 H, G, dim, vdim};
  const size_t smem = (size_t)(H + G) * dim * 4;
  if (smem > 96 * 1024) { dlti_set_error("qkv_rows: queries and keys of up to 24576 elements"); return DLTI_ERR_TOO_LARGE; }
  const bool vec = dtype == DLTI_BF16 && ((dim | vdim | oq | ok | ov | kd | vd | q_hd) & 7) == 0 && ((ld | f_ld | own_ld | q_ld) & 7) == 0 &&
                   ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(first) | reinterpret_cast<uintptr_t>(own) |
                     reinterpret_cast<uintptr_t>(kc) | reinterpret_cast<uintptr_t>(vc) | reinterpret_cast<uintptr_t>(q) |
                     reinterpret_cast<uintptr_t>(kp) | reinterpret_cast<uintptr_t>(vp)) & 15) == 0;
  using B = __nv_bfloat16;
  const int pieces = ((H + G) * dim + G * vdim) / 8;
  if (vec && pieces <= 128 * 12 &&
      ((reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(qn) | reinterpret_cast<uintptr_t>(kn)) & 15) == 0) {
    // a whole row's loads in flight: many threads in small steps, many rows in large ones
#define QR_CASE(V, TH)                                                                                                      \
  if (pieces <= TH * V) {                                                                                                   \
    auto kern = acc ? qkv_rows_vec_kernel<B, true, V, TH> : qkv_rows_vec_kernel<B, false, V, TH>;                            \
    DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, kern, dim3((unsigned)tokens), dim3(TH), 0, st, p));                              \
    dlti_count_launch();                                                                                                    \
    return 0;                                                                                                               \
  }
    if (tokens <= 512) { QR_CASE(1, 256) QR_CASE(1, 512) QR_CASE(2, 512) QR_CASE(3, 512) }
    QR_CASE(1, 128) QR_CASE(2, 128) QR_CASE(3, 128) QR_CASE(4, 128) QR_CASE(6, 128) QR_CASE(8, 128) QR_CASE(12, 128)
#undef QR_CASE
  }
  auto kern = vec ? (acc ? qkv_rows_kernel<B, true, 8> : qkv_rows_kernel<B, false, 8>)
                  : dtype == DLTI_BF16 ? (acc ? qkv_rows_kernel<B, true, 1> : qkv_rows_kernel<B, false, 1>)
                                       : (acc ? qkv_rows_kernel<float, true, 1> : qkv_rows_kernel<float, false, 1>);
  if (dtype != DLTI_BF16 && dtype != DLTI_FP32) return DLTI_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) DLTI_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, kern, dim3((unsigned)tokens), dim3(256), smem, st, p));
  dlti_count_launch();
  return 0;
}

DLTI_API int dlti_prefix_rows(void* packed, long long ld, int hd, const int* rows, const int* slots, const void* kc, const void* vc,
                              int kd, int vd, int H, int G, long long n, cudaStream_t st) {
  if (n <= 0) return 0;
  if (ld % 8 || hd % 8 || kd % 8 || vd % 8) return DLTI_ERR_BAD_ARG;
  const long long total = n * (H + 2 * G) * (hd / 8);
  prefix_rows_kernel<<<grid_for(total, 256), 256, 0, st>>>((__nv_bfloat16*)packed, ld, hd, rows, slots, (const __nv_bfloat16*)kc,
                                                           (const __nv_bfloat16*)vc, kd, vd, H, G, total);
  dlti_count_launch();
  return (int)cudaGetLastError();
}

DLTI_API int dlti_short_conv(const void* src, long long ld, int col, int C, int taps, const float* w, const float* b, int w_ld,
                             const void* state, const int* sslot, const int* rseq, const int* ctx, const int* cu, int nd, void* out,
                             long long o_ld, void* raw, long long raw_ld, int raw_n, float* tail, long long tail_ld, int tail0, long long rows,
                             int acc, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (taps < 1 || C < 1 || (tail && (!acc || tail0 % 8 || tail_ld % 4 || (reinterpret_cast<uintptr_t>(tail) & 15)))) return DLTI_ERR_BAD_ARG;
  ConvParams p{src, ld, col, C, taps, w, b, w_ld, state, sslot, rseq, ctx, cu, nd, out, o_ld, raw, raw_ld, raw_n, rows, tail, tail_ld, tail0};
  if (acc) {
    if (nd != rows || !raw || raw_n % 2) return DLTI_ERR_BAD_ARG;
    if (dtype == DLTI_BF16 && C % 8 == 0 && ld % 8 == 0 && col % 8 == 0 && raw_n % 8 == 0 && raw_ld % 8 == 0 && o_ld % 8 == 0 && w_ld % 4 == 0 &&
        ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(raw) | reinterpret_cast<uintptr_t>(w) |
          reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(state)) & 15) == 0) {
      DLTI_CUDA_CHECK(dlti_launch_pdl(rows, short_conv_acc_vec_kernel<__nv_bfloat16>, dim3((unsigned)rows, (raw_n / 8 + 127) / 128), dim3(128), 0,
                                      st, p));
      dlti_count_launch();
      return 0;
    }
    const int g = grid_for(rows * (raw_n / 2), 256);
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, short_conv_acc_kernel<T>, dim3(g), dim3(256), 0, st, p)));
  } else if (dtype == DLTI_BF16 && taps >= 2 && taps <= 4 && C % 8 == 0 && ld % 8 == 0 && col % 8 == 0 && o_ld % 8 == 0 && w_ld % 4 == 0 &&
             ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(w) |
               reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(state)) & 15) == 0) {
    using B = __nv_bfloat16;
    auto kern = taps == 2 ? short_conv_vec_kernel<B, 2> : taps == 3 ? short_conv_vec_kernel<B, 3> : short_conv_vec_kernel<B, 4>;
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kern, dim3((unsigned)((rows + CONV_ROWS - 1) / CONV_ROWS), (C / 8 + 127) / 128), dim3(128), 0, st, p));
  } else {
    const int g = grid_for(rows * ((C + 1) / 2), 256);
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, short_conv_kernel<T>, dim3(g), dim3(256), 0, st, p)));
  }
  dlti_count_launch();
  return 0;
}

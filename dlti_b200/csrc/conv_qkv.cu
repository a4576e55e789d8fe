// Merged attention projections -> queries, keys and values, head by head: a causal convolution over time on every channel, a norm per
// head of q and k, a factor on the queries by position, keys and values into the paged cache. The inputs of the last taps - 1 rows of a
// sequence are its state.
//
//   conv_qkv_vec     prompt rows, 16-bit, heads of 64, 128 or 256: lanes share a head and keep a window of rows in registers
//   conv_qkv_decode  one row per sequence from the decode GEMM's accumulator: the thread that reads a channel's state renews it; the
//                    output gates' columns are passed on
//   conv_qkv         any sizes, a warp per (row, head)
//   conv_state       renews the states where rows read one another's inputs (after the first kernel, and after the third on a
//                    projection in the activation type)
#include "rows.cuh"

namespace {

struct ConvQkv {
  const void* proj; long long ld;                          // merged projection rows
  int oq, ok, ov, og;                                      // section columns (og: only passed on from an accumulator; < 0: none)
  const float* w; int taps, w_ld;                          // tap-major weights by projection column (null: no convolution)
  void* state; int C;                                      // [slots, taps - 1, C]: inputs of the projection columns before the step
  const int *sslot, *rseq, *ctx, *cu; int nd;
  const float *qn, *kn; float eps;                         // per-head norm weights (null: no norm)
  const float* factors; const int* pos;                    // query factors by position (null: one)
  const long long* slots; void *kc, *vc; int kd, vd;       // cache row pitches of a head
  void* q; long long q_ld; int q_hd;                       // queries: row pitch, head pitch
  void *kp, *vp; const int* dst;                           // packed keys / values (row pitch q_ld, head pitch q_hd) or null; row of token t
                                                           // >= nd is nd + dst[t - nd] (dst null: t)
  void* gate; long long g_ld;
  long long tokens; int H, G, dim, vdim;
};
__device__ __forceinline__ long long out_row(const ConvQkv& p, long long t) { return (p.dst && t >= p.nd) ? p.nd + (long long)p.dst[t - p.nd] : t; }
// head `job` of a row: H queries, G keys, G values, then (gates) H
struct Job { int kind, head, col, n; };                    // kind 0 q, 1 k, 2 v, 3 gate
__device__ __forceinline__ Job job_of(const ConvQkv& p, int job) {
  if (job < p.H) return Job{0, job, p.oq + job * p.dim, p.dim};
  job -= p.H;
  if (job < p.G) return Job{1, job, p.ok + job * p.dim, p.dim};
  job -= p.G;
  if (job < p.G) return Job{2, job, p.ov + job * p.vdim, p.vdim};
  job -= p.G;
  return Job{3, job, p.og + job * p.vdim, p.vdim};
}

template <typename T, bool ACC, int MAXE>
__global__ void __launch_bounds__(128) conv_qkv_kernel(const ConvQkv p, int jobs) {
  griddep_wait();
  griddep_launch();
  const int lane = threadIdx.x & 31, hist = p.taps - 1;
  const long long total = p.tokens * jobs;
  for (long long x = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5; x < total; x += ((long long)gridDim.x * blockDim.x) >> 5) {
    const long long t = x / jobs;
    const Job job = job_of(p, (int)(x - t * jobs));
    const uint8_t* row = reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * (ACC ? 4 : sizeof(T));
    if (job.kind == 3) {
      T* g = reinterpret_cast<T*>(p.gate) + t * p.g_ld + (long long)job.head * p.vdim;
      for (int c = lane; c < job.n; c += 32) g[c] = Cvt<T>::from_f(take<T, ACC>(row, job.col + c));
      continue;
    }
    const long long slot = p.slots[t];
    const int s = p.rseq[t], sslot = hist > 0 && p.w ? p.sslot[s] : -1;
    long long row0;
    int n, start;
    seq_rows(p.cu, p.ctx, p.nd, s, row0, n, start);
    const int local = (int)(t - row0);
    float v[MAXE], ss = 0.f;
#pragma unroll
    for (int i = 0; i < MAXE; ++i) {
      const int e = lane + 32 * i, c = job.col + e;
      v[i] = 0.f;
      if (e < job.n) {
        const float u = take<T, ACC>(row, c);
        float a = u;
        if (p.w) {
          a = 0.f;
          T* st = reinterpret_cast<T*>(p.state) + (long long)sslot * hist * p.C + c - p.oq;
          for (int k = 0; k < hist; ++k) {
            const int r = local - hist + k;                // row of this tap relative to the step
            float in = 0.f;
            if (!ACC && r >= 0) in = Cvt<T>::to_f(reinterpret_cast<const T*>(p.proj)[(row0 + r) * p.ld + c]);
            else if (start > 0 && sslot >= 0) in = Cvt<T>::to_f(st[(long long)(r + hist) * p.C]);
            a = fmaf(p.w[(long long)k * p.w_ld + c - p.oq], in, a);
            if (ACC && sslot >= 0 && k > 0) st[(long long)(k - 1) * p.C] = Cvt<T>::from_f(in);
          }
          a = fmaf(p.w[(long long)hist * p.w_ld + c - p.oq], u, a);
          if (ACC && sslot >= 0) st[(long long)(hist - 1) * p.C] = Cvt<T>::from_f(u);
        }
        v[i] = a;
        ss += a * a;
      }
    }
    const float* nw = job.kind == 0 ? p.qn : job.kind == 1 ? p.kn : nullptr;
    ss = warp_sum(ss);
    float f = nw ? 1.f / sqrtf(ss / (float)job.n + p.eps) : 1.f;
    if (job.kind == 0 && p.factors) f *= p.factors[p.pos[t]];
    T *out, *cache = nullptr;
    if (job.kind == 0) {
      out = reinterpret_cast<T*>(p.q) + out_row(p, t) * p.q_ld + (long long)job.head * p.q_hd;
    } else {
      void* pk = job.kind == 1 ? p.kp : p.vp;
      out = pk ? reinterpret_cast<T*>(pk) + out_row(p, t) * p.q_ld + (long long)job.head * p.q_hd : nullptr;
      if (slot >= 0) cache = reinterpret_cast<T*>(job.kind == 1 ? p.kc : p.vc) + (slot * p.G + job.head) * (job.kind == 1 ? p.kd : p.vd);
    }
#pragma unroll
    for (int i = 0; i < MAXE; ++i) {
      const int e = lane + 32 * i;
      if (e < job.n) {
        const T o = Cvt<T>::from_f(v[i] * f * (nw ? nw[e] : 1.f));
        if (out) out[e] = o;
        if (cache) cache[e] = o;
      }
    }
  }
}

// 8 finished elements e0 ... of a head: norm over its LPH lanes (all lanes of the warp take part), factor, stores
template <typename T, int LPH>
__device__ __forceinline__ void finish(const ConvQkv& p, const Job& job, bool on, long long t, int e0, const float (&nw)[8], float (&a)[8]) {
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) ss += a[j] * a[j];
#pragma unroll
  for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!on) return;
  if (job.kind < 2) {
    float f = (job.kind == 0 ? p.qn : p.kn) ? rsqrtf(ss * (1.f / (8 * LPH)) + p.eps) : 1.f;
    if (job.kind == 0 && p.factors) f *= p.factors[p.pos[t]];
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] *= f * nw[j];
  }
  if (job.kind == 0) {
    put_n(reinterpret_cast<T*>(p.q) + out_row(p, t) * p.q_ld + job.head * p.q_hd + e0, a);
    return;
  }
  void* pk = job.kind == 1 ? p.kp : p.vp;
  const long long slot = p.slots[t];
  if (pk) put_n(reinterpret_cast<T*>(pk) + out_row(p, t) * p.q_ld + job.head * p.q_hd + e0, a);
  if (slot >= 0) put_n(reinterpret_cast<T*>(job.kind == 1 ? p.kc : p.vc) + (slot * p.G + job.head) * (job.kind == 1 ? p.kd : p.vd) + e0, a);
}
__device__ __forceinline__ void norm_weights(const ConvQkv& p, const Job& job, int e0, float (&nw)[8]) {
  const float* n = job.kind == 0 ? p.qn : job.kind == 1 ? p.kn : nullptr;
#pragma unroll
  for (int j = 0; j < 8; ++j) nw[j] = 1.f;
  if (n) ld8(n + e0, nw);
}

constexpr int CQ_ROWS = 8;                                 // rows of a thread's window
template <typename T, int LPH, int TAPS>
__global__ void __launch_bounds__(128) conv_qkv_vec_kernel(const ConvQkv p, int jobs) {
  constexpr int HPW = 32 / LPH, HIST = TAPS - 1;
  const int lane = threadIdx.x & 31, e0 = lane % LPH * 8;
  const int first = (blockIdx.y * 4 + (threadIdx.x >> 5)) * HPW, x = first + lane / LPH;
  if (first >= jobs) return;
  const bool on = x < jobs;
  const Job job = job_of(p, on ? x : jobs - 1);
  const int c = job.col + e0;
  float w[TAPS][8], nw[8];
  if (p.w) {
#pragma unroll
    for (int k = 0; k < TAPS; ++k) ld8(p.w + (long long)k * p.w_ld + c - p.oq, w[k]);
  } else {
#pragma unroll
    for (int k = 0; k < TAPS; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) w[k][j] = k == HIST ? 1.f : 0.f;
  }
  norm_weights(p, job, e0, nw);
  griddep_wait();
  griddep_launch();
  const long long t0 = (long long)blockIdx.x * CQ_ROWS;
  const int nr = (int)min((long long)CQ_ROWS, p.tokens - t0);
  const T* src = reinterpret_cast<const T*>(p.proj) + c;
  long long row0;
  int n, start;
  seq_rows(p.cu, p.ctx, p.nd, p.rseq[t0], row0, n, start);
  if (t0 - row0 >= HIST && t0 + nr <= row0 + n) {          // all inputs are rows of this step
    uint4 u[HIST + CQ_ROWS];                               // still packed: all loads in flight at half the registers
    const T* sp = src + (t0 - HIST) * p.ld;
#pragma unroll
    for (int i = 0; i < HIST + CQ_ROWS; ++i)
      if (i < HIST + nr) u[i] = *reinterpret_cast<const uint4*>(sp + i * p.ld);
#pragma unroll
    for (int r = 0; r < CQ_ROWS; ++r)
      if (r < nr) {
        float a[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] = 0.f;
#pragma unroll
        for (int k = 0; k < TAPS; ++k) {
          const uint32_t y[4] = {u[r + k].x, u[r + k].y, u[r + k].z, u[r + k].w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float2 f = Cvt<T>::unpack2(y[j]);
            a[2 * j] = fmaf(w[k][2 * j], f.x, a[2 * j]);
            a[2 * j + 1] = fmaf(w[k][2 * j + 1], f.y, a[2 * j + 1]);
          }
        }
        finish<T, LPH>(p, job, on, t0 + r, e0, nw, a);
      }
    return;
  }
  for (int r = 0; r < nr; ++r) {                           // a block with the start of a sequence: rows or state, tap by tap
    const long long t = t0 + r;
    const int s = p.rseq[t];
    seq_rows(p.cu, p.ctx, p.nd, s, row0, n, start);
    const int local = (int)(t - row0), slot = HIST > 0 ? p.sslot[s] : -1;
    float a[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] = 0.f;
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      const int q = local - HIST + k;
      float in[8];
      if (q >= 0) take_n<T, false, 8>(src + (row0 + q) * p.ld, 0, in);
      else if (start > 0 && slot >= 0) take_n<T, false, 8>(reinterpret_cast<const T*>(p.state) + ((long long)slot * HIST + q + HIST) * p.C + c - p.oq, 0, in);
      else continue;
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] = fmaf(w[k][j], in[j], a[j]);
    }
    finish<T, LPH>(p, job, on, t, e0, nw, a);
  }
}

template <typename T, int LPH>
__global__ void __launch_bounds__(128) conv_qkv_decode_kernel(const ConvQkv p, int jobs) {
  constexpr int HPW = 32 / LPH;
  const int lane = threadIdx.x & 31, e0 = lane % LPH * 8, hist = p.w ? p.taps - 1 : 0;
  const int first = (blockIdx.y * 4 + (threadIdx.x >> 5)) * HPW, x = first + lane / LPH;
  if (first >= jobs) return;
  const bool on = x < jobs;
  const Job job = job_of(p, on ? x : jobs - 1);
  const int c = job.col + e0;
  float a[8], w[8], nw[8];
  norm_weights(p, job, e0, nw);
  const bool conv = p.w && job.kind < 3;
  if (conv) ld8(p.w + (long long)hist * p.w_ld + c - p.oq, w);
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
#pragma unroll
  for (int j = 0; j < 8; ++j) a[j] = 0.f;
  if (on) take_n<T, true, 8>(reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * 4, c, a);
  if (job.kind == 3 && on) put_n(reinterpret_cast<T*>(p.gate) + t * p.g_ld + (long long)job.head * p.vdim + e0, a);
  if (conv && on) {
    const int slot = hist > 0 ? p.sslot[t] : -1;
    const bool have = slot >= 0 && p.ctx[t] > 1;
    T* st = reinterpret_cast<T*>(p.state) + (long long)slot * hist * p.C + c - p.oq;
    float u[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      u[j] = a[j];
      a[j] *= w[j];
    }
    for (int k = 0; k < hist; ++k) {
      float in[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) in[j] = 0.f;
      if (have) take_n<T, false, 8>(st + (long long)k * p.C, 0, in);
      ld8(p.w + (long long)k * p.w_ld + c - p.oq, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] = fmaf(w[j], in[j], a[j]);
      if (slot >= 0 && k > 0) put_n(st + (long long)(k - 1) * p.C, in);
    }
    if (slot >= 0) put_n(st + (long long)(hist - 1) * p.C, u);
  }
  finish<T, LPH>(p, job, on && job.kind < 3, t, e0, nw, a);
}

// the last taps - 1 inputs of every sequence become its state; entries move towards the front, so they may overwrite one another in order
template <typename T>
__global__ void __launch_bounds__(128) conv_state_kernel(const ConvQkv p) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x * 128 + threadIdx.x, s = blockIdx.y, hist = p.taps - 1;
  if (c >= p.C) return;
  const int slot = p.sslot[s];
  if (slot < 0) return;
  long long row0;
  int n, start;
  seq_rows(p.cu, p.ctx, p.nd, s, row0, n, start);
  if (n < 1) return;
  T* st = reinterpret_cast<T*>(p.state) + (long long)slot * hist * p.C + c;
  for (int k = 0; k < hist; ++k) {
    const int r = n - hist + k;
    T v = Cvt<T>::from_f(0.f);
    if (r >= 0) v = reinterpret_cast<const T*>(p.proj)[(row0 + r) * p.ld + p.oq + c];
    else if (start > 0) v = st[(long long)(r + hist) * p.C];
    st[(long long)k * p.C] = v;
  }
}

template <typename T, bool ACC>
int launch_general(const ConvQkv& p, int jobs, cudaStream_t st) {
  const int n = p.dim > p.vdim ? p.dim : p.vdim;
  if (n > 2048) { dlti_set_error("conv_qkv: heads of up to 2048 dimensions"); return DLTI_ERR_TOO_LARGE; }
  auto kern = n <= 128 ? conv_qkv_kernel<T, ACC, 4> : n <= 512 ? conv_qkv_kernel<T, ACC, 16> : conv_qkv_kernel<T, ACC, 64>;
  DLTI_CUDA_CHECK(dlti_launch_pdl(p.tokens, kern, dim3(grid_for(p.tokens * jobs * 32, 128)), dim3(128), 0, st, p, jobs));
  dlti_count_launch();
  return 0;
}

template <int LPH>
int launch_vec(const ConvQkv& p, int jobs, cudaStream_t st) {
  using B = __nv_bfloat16;
  const int per = 4 * (32 / LPH), taps = p.w ? p.taps : 1;
  auto kern = taps == 1 ? conv_qkv_vec_kernel<B, LPH, 1> : taps == 2 ? conv_qkv_vec_kernel<B, LPH, 2>
              : taps == 3 ? conv_qkv_vec_kernel<B, LPH, 3> : conv_qkv_vec_kernel<B, LPH, 4>;
  DLTI_CUDA_CHECK(dlti_launch_pdl(p.tokens, kern, dim3((unsigned)((p.tokens + CQ_ROWS - 1) / CQ_ROWS), (jobs + per - 1) / per), dim3(128), 0, st, p,
                                  jobs));
  dlti_count_launch();
  return 0;
}
template <int LPH>
int launch_decode(const ConvQkv& p, int jobs, cudaStream_t st) {
  const int per = 4 * (32 / LPH);
  DLTI_CUDA_CHECK(dlti_launch_pdl(p.tokens, conv_qkv_decode_kernel<__nv_bfloat16, LPH>, dim3((unsigned)p.tokens, (jobs + per - 1) / per), dim3(128),
                                  0, st, p, jobs));
  dlti_count_launch();
  return 0;
}

}  // namespace

// See ConvQkv. taps 0 or w null: no convolution. acc (rows = nd decode rows): proj is the decode GEMM's accumulator, zero on return, and the
// gate columns go to `gate`.
DLTI_API int dlti_conv_qkv(const void* proj, long long ld, int oq, int ok, int ov, int og, const float* w, int taps, int w_ld, void* state, int C,
                           const int* sslot, const int* rseq, const int* ctx, const int* cu, int nd, int nseq, const float* qn,
                           const float* kn, float eps, const float* factors, const int* pos, const long long* slots, void* kc, void* vc, int kd,
                           int vd, void* q, long long q_ld, int q_hd, void* kp, void* vp, const int* dst, void* gate, long long g_ld, long long tokens,
                           int H, int G, int dim, int vdim, int acc, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (H < 1 || G < 1 || H % G || dim < 1 || vdim < 1 || (w && taps < 1) || (w && taps > 1 && (!state || C < ov - oq + G * vdim)) ||
      (acc && (nd != tokens || (og >= 0 && !gate))) || nseq > 65535)
    return DLTI_ERR_BAD_ARG;
  if (!w) taps = 1;
  ConvQkv p{proj, ld, oq, ok, ov, og, w, taps, w_ld, state, C, sslot, rseq, ctx, cu, nd, qn, kn, eps, factors, pos, slots, kc, vc, kd, vd, q, q_ld, q_hd,
            kp, vp, dst, gate, g_ld, tokens, H, G, dim, vdim};
  const int jobs = H + 2 * G + (acc && og >= 0 ? H : 0);
  const uintptr_t all = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(state) |
                        reinterpret_cast<uintptr_t>(qn) | reinterpret_cast<uintptr_t>(kn) | reinterpret_cast<uintptr_t>(kc) |
                        reinterpret_cast<uintptr_t>(vc) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kp) |
                        reinterpret_cast<uintptr_t>(vp) | reinterpret_cast<uintptr_t>(gate);
  const bool vec = dtype == DLTI_BF16 && dim == vdim && (dim == 64 || dim == 128 || dim == 256) && (acc || taps <= 4) && (all & 15) == 0 &&
                   ((oq | ok | ov | (og < 0 ? 0 : og) | w_ld | C | kd | vd | q_hd) & 7) == 0 && ((ld | q_ld | g_ld) & 7) == 0 && tokens < (1ll << 31);
  int rc;
  if (vec && acc) return dim == 64 ? launch_decode<8>(p, jobs, st) : dim == 128 ? launch_decode<16>(p, jobs, st) : launch_decode<32>(p, jobs, st);
  if (vec) {
    rc = dim == 64 ? launch_vec<8>(p, jobs, st) : dim == 128 ? launch_vec<16>(p, jobs, st) : launch_vec<32>(p, jobs, st);
  } else if (acc) {
    DISPATCH_T(dtype, return (launch_general<T, true>(p, jobs, st)));
  } else {
    DISPATCH_T(dtype, rc = (launch_general<T, false>(p, jobs, st)));
  }
  if (rc) return rc;
  if (taps > 1) {
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, conv_state_kernel<T>, dim3((C + 127) / 128, (unsigned)nseq), dim3(128), 0, st, p)));
    dlti_count_launch();
  }
  return 0;
}

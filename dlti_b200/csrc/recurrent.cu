// Linear recurrences with an outer-product update, one state matrix per head:
//     S_t = a_t S_(t-1) + k_t (s_t v_t)^T,      o_t = S_t^T q_t + D v_t        (S is N x P, fp32)
// Mamba-2:    k = B, q = C (shared by the heads of a group), v = x, s_t = dt, a_t = exp(-exp(A_log) dt), D per head
// lightning:  a_t = one constant per head, s_t = 1, D = 0, silu on q, k, v as they are loaded
// States live in slots [slots, heads, N, P] and are carried from step to step; a sequence whose step starts at position
// 0 starts from zero whatever its slot holds.
#include "common.cuh"

namespace {

struct ScanParams {
  const void *q, *k, *v;
  long long q_ld, k_ld, v_ld;
  int rep;                                 // heads per q/k group
  int silu;
  const float* decay;                  // [heads] or null
  const void* dt; long long dt_ld;         // raw step sizes [rows, heads] (T) when decay is null
  const float *dt_bias, *A_log, *D;        // [heads]; D may be null
  float* state;
  const int *sslot, *ctx, *cu;
  int nd, seq0, heads, N, P;
  void* out; long long o_ld;
  // tail job: new convolution state = last conv_rows inputs of every sequence
  const void* conv_src; long long conv_ld; int conv_col, conv_rows, conv_C;
  void* conv_state;
};

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

__device__ __forceinline__ void seq_rows(const ScanParams& p, int s, long long& row0, int& n, int& start) {
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
template <typename T>
__device__ __forceinline__ void conv_tail(const ScanParams& p, int s, int part, int parts) {
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

// Token-by-token form. CTA = (32 columns of P, head, sequence), 8 warps: lane = column, a warp owns the NR consecutive
// rows [warp * NR, ...), so q and k are warp-uniform shared-memory reads. TT tokens are staged at a time; the warps'
// partial outputs are summed once per stage.
constexpr int TT = 8;
template <typename T, int NR>
__global__ void __launch_bounds__(256) scan_kernel(const ScanParams p, int slices, int conv_parts) {
  griddep_wait();
  griddep_launch();
  const int s = p.seq0 + blockIdx.z;
  if ((int)blockIdx.x >= slices) {
    if (blockIdx.y == 0) conv_tail<T>(p, s, blockIdx.x - slices, conv_parts);
    return;
  }
  __shared__ float sk[TT][8 * NR], sq[TT][8 * NR], sv[TT][32], part[TT][8][32], sa[TT];
  long long row0;
  int n, start;
  seq_rows(p, s, row0, n, start);
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col = blockIdx.x * 32 + lane, grp = h / p.rep;
  const int slot = p.sslot[s];
  const bool colok = col < p.P;
  float* st = p.state + (((long long)(slot < 0 ? 0 : slot) * p.heads + h) * p.N) * p.P + col;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = warp * NR + i;
    S[i] = (slot >= 0 && start > 0 && colok && r < p.N) ? st[(long long)r * p.P] : 0.f;
  }
  const float Dh = p.D ? p.D[h] : 0.f;
  const float cdec = p.decay ? p.decay[h] : 0.f;
  const T* q = reinterpret_cast<const T*>(p.q) + (long long)grp * p.N;
  const T* k = reinterpret_cast<const T*>(p.k) + (long long)grp * p.N;
  const T* v = reinterpret_cast<const T*>(p.v) + (long long)h * p.P;
  for (int t0 = 0; t0 < n; t0 += TT) {
    const int nt = min(TT, n - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * 8 * NR; i += 256) {
      const int t = i / (8 * NR), r = i - t * (8 * NR);
      const long long row = row0 + t0 + t;
      float kv = 0.f, qv = 0.f;
      if (r < p.N) {
        kv = Cvt<T>::to_f(k[row * p.k_ld + r]);
        qv = Cvt<T>::to_f(q[row * p.q_ld + r]);
        if (p.silu) { kv = Cvt<T>::to_f(Cvt<T>::from_f(silu_f(kv))); qv = Cvt<T>::to_f(Cvt<T>::from_f(silu_f(qv))); }
      }
      sk[t][r] = kv;
      sq[t][r] = qv;
    }
    if (warp < nt) {
      const long long row = row0 + t0 + warp;
      float x = colok ? Cvt<T>::to_f(v[row * p.v_ld + col]) : 0.f;
      if (p.silu) x = Cvt<T>::to_f(Cvt<T>::from_f(silu_f(x)));
      sv[warp][lane] = x;
      if (lane == 0) {
        if (p.decay) {
          sa[warp] = 1.f;
        } else {
          sa[warp] = softplus_f(Cvt<T>::to_f(reinterpret_cast<const T*>(p.dt)[row * p.dt_ld + h]) + p.dt_bias[h]);
        }
      }
    }
    __syncthreads();
    const float eA = p.decay ? 0.f : expf(p.A_log[h]);
    for (int t = 0; t < nt; ++t) {
      const float sc = sa[t];
      const float a = p.decay ? cdec : expf(-eA * sc);
      const float vv = sv[t][lane] * sc;
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        S[i] = fmaf(a, S[i], sk[t][warp * NR + i] * vv);
        acc = fmaf(sq[t][warp * NR + i], S[i], acc);
      }
      part[t][warp][lane] = acc;
    }
    __syncthreads();
    if (warp < nt && colok) {
      float o = Dh * sv[warp][lane];
#pragma unroll
      for (int w = 0; w < 8; ++w) o += part[warp][w][lane];
      reinterpret_cast<T*>(p.out)[(row0 + t0 + warp) * p.o_ld + (long long)h * p.P + col] = Cvt<T>::from_f(o);
    }
  }
  if (slot >= 0 && colok) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = warp * NR + i;
      if (r < p.N) st[(long long)r * p.P] = S[i];
    }
  }
}

template <typename T>
int launch_scan(const ScanParams& p, int nseq, cudaStream_t st) {
  const int slices = (p.P + 31) / 32;
  const int conv_parts = p.conv_state ? (p.conv_C + 2047) / 2048 : 0;
  const dim3 grid(slices + conv_parts, p.heads, nseq);
  const long long rows = p.nd;                 // a programmatic dependent launch only pays in decode-sized steps
#define SCAN_CASE(NR)                                                                                                         \
  if (p.N <= 8 * NR) {                                                                                                        \
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows > 0 && p.seq0 + nseq <= p.nd ? rows : 1 << 20, scan_kernel<T, NR>, grid, dim3(256), 0, st, \
                                    p, slices, conv_parts));                                                                  \
    dlti_count_launch();                                                                                                      \
    return 0;                                                                                                                 \
  }
  SCAN_CASE(4) SCAN_CASE(8) SCAN_CASE(16) SCAN_CASE(32)
#undef SCAN_CASE
  dlti_set_error("linear_scan: states of up to 256 rows");
  return DLTI_ERR_TOO_LARGE;
}

}  // namespace

// Sequences [seq0, seq0 + nseq) of the step (the first nd sequences are single rows, sequence nd + i has the rows
// nd + cu[i] ... nd + cu[i + 1]). conv_state: optional tail job, see conv_tail.
DLTI_API int dlti_linear_scan(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, int rep,
                              int silu, const float* decay, const void* dt, long long dt_ld, const float* dt_bias,
                              const float* A_log, const float* D, float* state, const int* sslot, const int* ctx, const int* cu, int nd,
                              int seq0, int nseq, int heads, int N, int P, void* out, long long o_ld, const void* conv_src,
                              long long conv_ld, int conv_col, int conv_rows, int conv_C, void* conv_state, int dtype,
                              cudaStream_t st) {
  if (nseq <= 0) return 0;
  if (heads < 1 || rep < 1 || N < 1 || P < 1 || nseq > 65535 || (!decay && (!dt || !dt_bias || !A_log))) return DLTI_ERR_BAD_ARG;
  if (conv_rows <= 0) conv_state = nullptr;
  ScanParams p{q, k, v, q_ld, k_ld, v_ld, rep, silu, decay, dt, dt_ld, dt_bias, A_log, D, state, sslot, ctx, cu,
               nd, seq0, heads, N, P, out, o_ld, conv_src, conv_ld, conv_col, conv_rows, conv_C, conv_state};
  if (dtype == DLTI_BF16) return launch_scan<__nv_bfloat16>(p, nseq, st);
  if (dtype == DLTI_FP32) return launch_scan<float>(p, nseq, st);
  return DLTI_ERR_UNSUPPORTED;
}

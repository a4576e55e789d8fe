// Row kernels of pre-norm layers on several residual streams (hyper-connections), each sublayer behind a layer norm and a
// short causal convolution of its input, and the PolyNorm activation.
//
// A token's streams lie next to each other, x [rows, S, d] fp32. Between two sublayers one kernel does everything a row
// needs: x_t <- sum_s mix[s, t] x_s + out[t] y with the finished sublayer's output y, then h = layer_norm(sum_s in[s] x_s) w
// for the next one; with one token per sequence also the input convolution and its state. The convolution of prompt rows
// reads neighbouring rows and is a kernel of its own.
#include "rows.cuh"

namespace {

struct HyperParams {
  float* x; int S, d;
  const void* y; long long y_ld;                           // finished sublayer's output (null: streams stay)
  const float *mix, *out;                                  // [S, S] from, to; [S]
  const float *in, *w; float eps;                          // [S] (null: plain sum), [d] (w null: nothing is read)
  const float* cw; int cw_ld, taps;                        // tap-major convolution weights (null: none)
  void* cstate; const int *sslot, *ctx;                    // [slots, taps - 1, d]; row t is sequence t
  void* h; long long h_ld;
  const long long* idx;                                    // rows to read (only without y)
};

// h + conv(h) of one row's channels c .. c + N - 1 whose earlier inputs are the state; the state moves on by one
template <typename T, int N>
__device__ __forceinline__ void canon_step(const HyperParams& p, int slot, bool hist, int c, float (&h)[N]) {
  float a[N];
#pragma unroll
  for (int j = 0; j < N; ++j) a[j] = 0.f;
  T* st = reinterpret_cast<T*>(p.cstate) + (long long)slot * (p.taps - 1) * p.d + c;
  for (int k = 0; k < p.taps - 1; ++k) {
    float x[N];
#pragma unroll
    for (int j = 0; j < N; ++j) x[j] = 0.f;
    if (slot >= 0) {
      if (hist) take_n<T, false, N>(st + (long long)k * p.d, 0, x);
      if (k > 0) put_n<T, N>(st + (long long)(k - 1) * p.d, x);
    }
#pragma unroll
    for (int j = 0; j < N; ++j) a[j] += p.cw[(long long)k * p.cw_ld + c + j] * x[j];
  }
#pragma unroll
  for (int j = 0; j < N; ++j) h[j] = round_to<T>(h[j]);
  if (slot >= 0 && p.taps > 1) put_n<T, N>(st + (long long)(p.taps - 2) * p.d, h);
#pragma unroll
  for (int j = 0; j < N; ++j) h[j] += a[j] + p.cw[(long long)(p.taps - 1) * p.cw_ld + c + j] * h[j];
}

template <typename T, bool ACC, int S, int VPT>
__global__ void __launch_bounds__(512) hyper_vec_kernel(const HyperParams p) {
  __shared__ float red[32];
  const int vec = p.d >> 2;
  float mix[S][S], wo[S], wi[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {                            // weights never change: they may come before the wait
    wi[s] = p.in ? p.in[s] : 1.f;
    wo[s] = p.y ? p.out[s] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = p.y ? p.mix[s * S + t] : 0.f;
  }
  griddep_wait();
  griddep_launch();
  const long long row = p.idx ? p.idx[blockIdx.x] : (long long)blockIdx.x;
  float* xr = p.x + row * S * p.d;
  const void* yr = reinterpret_cast<const uint8_t*>(p.y) + row * p.y_ld * (ACC ? 4 : sizeof(T));
  float u[VPT][4];
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
#pragma unroll
    for (int j = 0; j < 4; ++j) u[i][j] = 0.f;
    if (v >= vec) continue;
    float x[S][4];
#pragma unroll
    for (int s = 0; s < S; ++s) *reinterpret_cast<float4*>(x[s]) = *reinterpret_cast<const float4*>(xr + (long long)s * p.d + v * 4);
    if (p.y) {
      float y[4], n[S][4];
      take_n<T, ACC, 4>(yr, v * 4, y);
#pragma unroll
      for (int t = 0; t < S; ++t) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          n[t][j] = wo[t] * y[j];
#pragma unroll
          for (int s = 0; s < S; ++s) n[t][j] = fmaf(mix[s][t], x[s][j], n[t][j]);
        }
        *reinterpret_cast<float4*>(xr + (long long)t * p.d + v * 4) = *reinterpret_cast<const float4*>(n[t]);
      }
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int j = 0; j < 4; ++j) x[s][j] = n[s][j];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
      for (int s = 0; s < S; ++s) u[i][j] = fmaf(wi[s], x[s][j], u[i][j]);
      sum += u[i][j];
    }
  }
  if (!p.w) return;
  const float mean = block_sum(sum, red) / (float)p.d;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (threadIdx.x + i * blockDim.x < vec)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        u[i][j] -= mean;
        ss += u[i][j] * u[i][j];
      }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)p.d + p.eps);
  const int slot = p.cw ? p.sslot[row] : -1;
  const bool hist = p.cw && p.ctx[row] > 1;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= vec) continue;
    const float4 w = *reinterpret_cast<const float4*>(p.w + v * 4);
    float h[4] = {u[i][0] * r * w.x, u[i][1] * r * w.y, u[i][2] * r * w.z, u[i][3] * r * w.w};
    if (p.cw) canon_step<T, 4>(p, slot, hist, v * 4, h);
    put_n<T, 4>(reinterpret_cast<T*>(p.h) + (long long)blockIdx.x * p.h_ld + v * 4, h);
  }
}

// any width, up to HYPER_MAX streams
constexpr int HYPER_MAX = 16;
template <typename T, bool ACC>
__global__ void __launch_bounds__(256) hyper_kernel(const HyperParams p) {
  __shared__ float red[32];
  extern __shared__ float u[];                             // [d]; a thread only touches its own channels
  griddep_wait();
  griddep_launch();
  const int S = p.S;
  const long long row = p.idx ? p.idx[blockIdx.x] : (long long)blockIdx.x;
  float* xr = p.x + row * S * p.d;
  const void* yr = reinterpret_cast<const uint8_t*>(p.y) + row * p.y_ld * (ACC ? 4 : sizeof(T));
  float sum = 0.f;
  for (int c = threadIdx.x; c < p.d; c += blockDim.x) {
    float x[HYPER_MAX];
    for (int s = 0; s < S; ++s) x[s] = xr[(long long)s * p.d + c];
    float a = 0.f;
    if (p.y) {
      const float y = take<T, ACC>(yr, c);
      for (int t = 0; t < S; ++t) {
        float n = p.out[t] * y;
        for (int s = 0; s < S; ++s) n = fmaf(p.mix[s * S + t], x[s], n);
        xr[(long long)t * p.d + c] = n;
        a = fmaf(p.in ? p.in[t] : 1.f, n, a);
      }
    } else {
      for (int s = 0; s < S; ++s) a = fmaf(p.in ? p.in[s] : 1.f, x[s], a);
    }
    u[c] = a;
    sum += a;
  }
  if (!p.w) return;
  const float mean = block_sum(sum, red) / (float)p.d;
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.d; c += blockDim.x) ss += (u[c] - mean) * (u[c] - mean);
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)p.d + p.eps);
  const int slot = p.cw ? p.sslot[row] : -1;
  const bool hist = p.cw && p.ctx[row] > 1;
  T* hr = reinterpret_cast<T*>(p.h) + (long long)blockIdx.x * p.h_ld;
  for (int c = threadIdx.x; c < p.d; c += blockDim.x) {
    float h = (u[c] - mean) * r * p.w[c];
    if (p.cw) {
      float a = 0.f;
      T* st = reinterpret_cast<T*>(p.cstate) + (long long)slot * (p.taps - 1) * p.d + c;
      for (int k = 0; k < p.taps - 1; ++k) {
        float x = 0.f;
        if (slot >= 0) {
          if (hist) x = Cvt<T>::to_f(st[(long long)k * p.d]);
          if (k > 0) st[(long long)(k - 1) * p.d] = Cvt<T>::from_f(x);
        }
        a += p.cw[(long long)k * p.cw_ld + c] * x;
      }
      h = round_to<T>(h);
      if (slot >= 0 && p.taps > 1) st[(long long)(p.taps - 2) * p.d] = Cvt<T>::from_f(h);
      h += a + p.cw[(long long)(p.taps - 1) * p.cw_ld + c] * h;
    }
    hr[c] = Cvt<T>::from_f(h);
  }
}

template <typename T, bool ACC>
int launch_hyper(const HyperParams& p, long long rows, cudaStream_t st) {
  const uintptr_t al = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.w) |
                       reinterpret_cast<uintptr_t>(p.h) | reinterpret_cast<uintptr_t>(p.cstate);
  if (p.d % 4 == 0 && p.d <= 8192 && p.S <= 4 && p.y_ld % 4 == 0 && p.h_ld % 4 == 0 && (al & 15) == 0) {
    const int vec = p.d / 4, vpt = vec <= 512 ? 1 : (vec <= 1024 ? 2 : 4);
    const int threads = ((vec + vpt - 1) / vpt + 31) / 32 * 32;
#define HV(S, V) hyper_vec_kernel<T, ACC, S, V>
#define HVS(V) (p.S == 1 ? HV(1, V) : p.S == 2 ? HV(2, V) : p.S == 3 ? HV(3, V) : HV(4, V))
    auto kern = vpt == 1 ? HVS(1) : vpt == 2 ? HVS(2) : HVS(4);
#undef HVS
#undef HV
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kern, dim3((unsigned)rows), dim3(threads), 0, st, p));
  } else {
    const size_t smem = (size_t)p.d * 4;
    if (p.S > HYPER_MAX || smem > 47 * 1024) { dlti_set_error("hyper: up to 16 streams of up to 12032 channels"); return DLTI_ERR_TOO_LARGE; }
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, hyper_kernel<T, ACC>, dim3((unsigned)rows), dim3(256), smem, st, p));
  }
  dlti_count_launch();
  return 0;
}

// x[t, s] = table[ids[t]] * scale for every stream s
template <typename T>
__global__ void embed_streams_kernel(const long long* __restrict__ ids, const T* __restrict__ table, float* __restrict__ x, long long tokens,
                                     int S, int d, long long vocab, float scale) {
  griddep_wait();
  griddep_launch();
  const long long total = tokens * d;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / d;
    const int c = (int)(i - t * d);
    const long long id = ids[t];
    const float v = (id >= 0 && id < vocab) ? Cvt<T>::to_f(table[id * d + c]) * scale : 0.f;
    for (int s = 0; s < S; ++s) x[(t * S + s) * d + c] = v;
  }
}

// out = h + conv(h) over the rows of the sequences seq0 + blockIdx.z; a block takes R >= taps - 1 consecutive rows of one
// sequence, so only its first block reads the state of earlier steps, and that block renews it afterwards.
struct CanonParams {
  const void* h; long long h_ld; int d, taps;
  const float* w; int w_ld;
  void* state; const int *sslot, *ctx, *cu; int nd, seq0;
  void* out; long long o_ld;
  int R;
};
template <typename T>
__global__ void __launch_bounds__(128) canon_kernel(const CanonParams p) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.y * 128 + threadIdx.x, s = p.seq0 + blockIdx.z, hist = p.taps - 1;
  long long row0;
  int n, start;
  seq_rows(p.cu, p.ctx, p.nd, s, row0, n, start);
  const int r0 = blockIdx.x * p.R, r1 = min(n, r0 + p.R);
  if (c >= p.d || r0 >= n) return;
  const T* h = reinterpret_cast<const T*>(p.h) + row0 * p.h_ld + c;
  const int slot = p.sslot[s];
  T* st = reinterpret_cast<T*>(p.state) + (long long)(slot < 0 ? 0 : slot) * hist * p.d + c;
  const bool have = slot >= 0 && start > 0;
  for (int r = r0; r < r1; ++r) {
    float a = 0.f;
    for (int k = 0; k < p.taps; ++k) {
      const int q = r - hist + k;
      const float x = q >= 0 ? Cvt<T>::to_f(h[(long long)q * p.h_ld]) : (have ? Cvt<T>::to_f(st[(long long)(q + hist) * p.d]) : 0.f);
      a += p.w[(long long)k * p.w_ld + c] * x;
    }
    reinterpret_cast<T*>(p.out)[(row0 + r) * p.o_ld + c] = Cvt<T>::from_f(Cvt<T>::to_f(h[(long long)r * p.h_ld]) + a);
  }
  if (r0 == 0 && slot >= 0)
    for (int j = 0; j < hist; ++j) {                       // entry j <- the input at row n - hist + j (an older one has a higher index)
      const int q = n - hist + j;
      st[(long long)j * p.d] = q >= 0 ? h[(long long)q * p.h_ld] : (have ? st[(long long)(q + hist) * p.d] : Cvt<T>::from_f(0.f));
    }
}
// the same, 8 channels a thread with the window in registers (16-bit T; d and pitches multiples of 8; TAPS fixed)
constexpr int CANON_ROWS = 8;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) canon_vec_kernel(const CanonParams p) {
  griddep_wait();
  griddep_launch();
  const int cv = blockIdx.y * 128 + threadIdx.x, s = p.seq0 + blockIdx.z;
  long long row0;
  int n, start;
  seq_rows(p.cu, p.ctx, p.nd, s, row0, n, start);
  const int r0 = blockIdx.x * CANON_ROWS, nr = min(CANON_ROWS, n - r0);
  if (cv >= (p.d >> 3) || nr <= 0) return;
  const int c = cv * 8;
  const T* h = reinterpret_cast<const T*>(p.h) + row0 * p.h_ld + c;
  const int slot = p.sslot[s];
  T* st = reinterpret_cast<T*>(p.state) + (long long)(slot < 0 ? 0 : slot) * (TAPS - 1) * p.d + c;
  const bool have = slot >= 0 && start > 0;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 x[TAPS - 1 + CANON_ROWS];                          // packed: all loads in flight
#pragma unroll
  for (int i = 0; i < TAPS - 1 + CANON_ROWS; ++i) {
    const int q = r0 - (TAPS - 1) + i;
    if (i < TAPS - 1 && q < 0) x[i] = have ? *reinterpret_cast<const uint4*>(st + (long long)(q + TAPS - 1) * p.d) : zero;
    else if (i < TAPS - 1 + nr) x[i] = *reinterpret_cast<const uint4*>(h + (long long)q * p.h_ld);
  }
  uint4 keep[TAPS - 1];
  if (r0 == 0 && slot >= 0)
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int q = n - (TAPS - 1) + j;
      keep[j] = q >= 0 ? *reinterpret_cast<const uint4*>(h + (long long)q * p.h_ld) : zero;
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i)                   // rows before the step: state entry q + TAPS - 1
        if (q < 0 && i == q + TAPS - 1) keep[j] = x[i];
    }
  float w[TAPS][8];
#pragma unroll
  for (int k = 0; k < TAPS; ++k) ld8(p.w + (long long)k * p.w_ld + c, w[k]);
#pragma unroll
  for (int r = 0; r < CANON_ROWS; ++r)
    if (r < nr) {
      float a[8], f[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] = 0.f;
#pragma unroll
      for (int k = 0; k < TAPS; ++k) {
        const uint32_t u[4] = {x[r + k].x, x[r + k].y, x[r + k].z, x[r + k].w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 v = Cvt<T>::unpack2(u[j]);
          f[2 * j] = v.x; f[2 * j + 1] = v.y;
          a[2 * j] += w[k][2 * j] * v.x;
          a[2 * j + 1] += w[k][2 * j + 1] * v.y;
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] += f[j];
      put_n<T, 8>(reinterpret_cast<T*>(p.out) + (row0 + r0 + r) * p.o_ld + c, a);
    }
  if (r0 == 0 && slot >= 0)
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) *reinterpret_cast<uint4*>(st + (long long)j * p.d) = keep[j];
}

// out = a N(z) + b N(z^2) + c N(z^3) + e over each row, N(y) = y / sqrt(mean y^2 + eps); coef = {a, b, c, e}
__device__ __forceinline__ float3 block_sum3(float3 v, float* red) {
  v.x = warp_sum(v.x); v.y = warp_sum(v.y); v.z = warp_sum(v.z);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (l == 0) { red[w] = v.x; red[32 + w] = v.y; red[64 + w] = v.z; }
  __syncthreads();
  return make_float3(warp_sum(l < nw ? red[l] : 0.f), warp_sum(l < nw ? red[32 + l] : 0.f), warp_sum(l < nw ? red[64 + l] : 0.f));
}
template <typename T, bool ACC, int VPT, int NT>
__global__ void __launch_bounds__(NT) poly_norm_vec_kernel(const void* __restrict__ z, long long z_ld, const float* __restrict__ coef,
                                                            T* __restrict__ out, long long o_ld, int n, float eps) {
  __shared__ float red[96];
  const float a = coef[0], b = coef[1], c = coef[2], e = coef[3];
  griddep_wait();
  griddep_launch();
  const long long row = blockIdx.x;
  const void* zr = reinterpret_cast<const uint8_t*>(z) + row * z_ld * (ACC ? 4 : sizeof(T));
  const int vec = n >> 3;
  float f[VPT][8];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < vec) take_n<T, ACC, 8>(zr, v * 8, f[i]);
  }
  float3 s = make_float3(0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (threadIdx.x + i * blockDim.x < vec)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float q = f[i][j] * f[i][j], q2 = q * q;
        s.x += q;
        s.y += q2;
        s.z += q2 * q;
      }
  s = block_sum3(s, red);
  const float ra = a / sqrtf(s.x / (float)n + eps), rb = b / sqrtf(s.y / (float)n + eps), rc = c / sqrtf(s.z / (float)n + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= vec) continue;
#pragma unroll
    for (int j = 0; j < 8; ++j) f[i][j] = fmaf(fmaf(fmaf(rc, f[i][j], rb), f[i][j], ra), f[i][j], e);
    put_n<T, 8>(out + row * o_ld + v * 8, f[i]);
  }
}
template <typename T, bool ACC>
__global__ void __launch_bounds__(256) poly_norm_kernel(const void* __restrict__ z, long long z_ld, const float* __restrict__ coef,
                                                        T* __restrict__ out, long long o_ld, int n, float eps) {
  __shared__ float red[96];
  extern __shared__ float row_s[];
  griddep_wait();
  griddep_launch();
  const long long row = blockIdx.x;
  const void* zr = reinterpret_cast<const uint8_t*>(z) + row * z_ld * (ACC ? 4 : sizeof(T));
  float3 s = make_float3(0.f, 0.f, 0.f);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float v = row_s[i] = take<T, ACC>(zr, i);
    const float q = v * v, q2 = q * q;
    s.x += q;
    s.y += q2;
    s.z += q2 * q;
  }
  s = block_sum3(s, red);
  const float ra = coef[0] / sqrtf(s.x / (float)n + eps), rb = coef[1] / sqrtf(s.y / (float)n + eps), rc = coef[2] / sqrtf(s.z / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float v = row_s[i];
    out[row * o_ld + i] = Cvt<T>::from_f(fmaf(fmaf(fmaf(rc, v, rb), v, ra), v, coef[3]));
  }
}

// columns [0, split) of the decode GEMM's accumulator as T, columns [split, n) as fp32; the accumulator becomes zero
template <typename T>
__global__ void split_rows_kernel(float* __restrict__ acc, T* __restrict__ out, long long o_ld, float* __restrict__ tail, long long t_ld,
                                  long long rows, int n, int split) {
  griddep_wait();
  griddep_launch();
  const int vec = n >> 3;
  const long long total = rows * vec;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / vec;
    const int c = 8 * (int)(i - r * vec);
    float f[8];
    float* src = acc + r * n + c;
    ld8(src, f);
    const float z[8] = {};
    st8(src, z);
    if (c < split) put_n<T, 8>(out + r * o_ld + c, f);
    else st8(tail + r * t_ld + c - split, f);
  }
}

}  // namespace

// y != null: streams [rows, S, d] are renewed from the sublayer output y (its fp32 accumulator with acc, zero on return).
// w != null: h [rows (of idx)] = layer_norm(sum_s in[s] x_s) * w; cw != null (row t is the newest token of sequence t): plus
// its causal convolution over the inputs kept in cstate.
DLTI_API int dlti_hyper(float* x, int S, int d, const void* y, long long y_ld, const float* mix, const float* out, const float* in,
                        const float* w, float eps, const float* cw, int cw_ld, int taps, void* cstate, const int* sslot, const int* ctx,
                        void* h, long long h_ld, const long long* idx, long long rows, int acc, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (S < 1 || d < 1 || (y && (!mix || !out || idx)) || (w && !h) || (cw && (!w || !sslot || !ctx || taps < 1 || (taps > 1 && !cstate)))) return DLTI_ERR_BAD_ARG;
  HyperParams p{x, S, d, y, y ? y_ld : 0, mix, out, in, w, eps, cw, cw_ld, taps, cstate, sslot, ctx, h, h_ld, idx};
  if (acc && dtype != DLTI_BF16) return DLTI_ERR_UNSUPPORTED;
  if (acc) return launch_hyper<__nv_bfloat16, true>(p, rows, st);
  DISPATCH_T(dtype, return (launch_hyper<T, false>(p, rows, st)));
}

DLTI_API int dlti_embed_streams(const long long* ids, const void* table, float* x, long long tokens, int S, int d, long long vocab,
                                float scale, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, embed_streams_kernel<T>, dim3(grid_for(tokens * d, 256)), dim3(256), 0, st, ids,
                                                    (const T*)table, x, tokens, S, d, vocab, scale)));
  dlti_count_launch();
  return 0;
}

// out = h + causal convolution of h; sequences seq0 ... seq0 + nseq - 1 of the step with at most max_rows rows each; the
// state [slots, taps - 1, d] is read and renewed.
DLTI_API int dlti_canon(const void* h, long long h_ld, int d, int taps, const float* w, int w_ld, void* state, const int* sslot,
                        const int* ctx, const int* cu, int nd, int seq0, int nseq, int max_rows, void* out, long long o_ld, int dtype,
                        cudaStream_t st) {
  if (nseq <= 0 || max_rows <= 0) return 0;
  if (taps < 1 || d < 1 || nseq > 65535 || h == out) return DLTI_ERR_BAD_ARG;
  CanonParams p{h, h_ld, d, taps, w, w_ld, state, sslot, ctx, cu, nd, seq0, out, o_ld, taps - 1 > 8 ? taps - 1 : 8};
  const uintptr_t al = reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(state);
  const long long pdl = (long long)max_rows * nseq;
  if (dtype == DLTI_BF16 && taps >= 2 && taps <= 4 && d % 8 == 0 && h_ld % 8 == 0 && o_ld % 8 == 0 && w_ld % 4 == 0 && (al & 15) == 0) {
    using B = __nv_bfloat16;
    auto kern = taps == 2 ? canon_vec_kernel<B, 2> : taps == 3 ? canon_vec_kernel<B, 3> : canon_vec_kernel<B, 4>;
    DLTI_CUDA_CHECK(dlti_launch_pdl(pdl, kern, dim3((max_rows + CANON_ROWS - 1) / CANON_ROWS, (d / 8 + 127) / 128, nseq), dim3(128), 0, st, p));
  } else {
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(pdl, canon_kernel<T>, dim3((max_rows + p.R - 1) / p.R, (d + 127) / 128, nseq), dim3(128), 0,
                                                      st, p)));
  }
  dlti_count_launch();
  return 0;
}

DLTI_API int dlti_poly_norm(const void* z, long long z_ld, const float* coef, void* out, long long o_ld, long long rows, int n, float eps,
                            int acc, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (acc && dtype != DLTI_BF16) return DLTI_ERR_UNSUPPORTED;
  if (dtype == DLTI_BF16 && n % 8 == 0 && n <= 16384 && z_ld % 8 == 0 && o_ld % 8 == 0 &&
      ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15) == 0) {
    using B = __nv_bfloat16;
    const int vec = n / 8, most = rows <= 256 ? 1024 : 256;          // few rows: all of a row's loads at once
    const int vpt = vec <= most ? 1 : vec <= 2 * most ? 2 : vec <= 4 * most ? 4 : 8, threads = ((vec + vpt - 1) / vpt + 31) / 32 * 32;
#define PV(AC) (most == 1024 ? (vpt == 1 ? poly_norm_vec_kernel<B, AC, 1, 1024> : poly_norm_vec_kernel<B, AC, 2, 1024>)   \
                : vpt == 1 ? poly_norm_vec_kernel<B, AC, 1, 256> : vpt == 2 ? poly_norm_vec_kernel<B, AC, 2, 256>       \
                : vpt == 4 ? poly_norm_vec_kernel<B, AC, 4, 256> : poly_norm_vec_kernel<B, AC, 8, 256>)
    auto kern = acc ? PV(true) : PV(false);
#undef PV
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kern, dim3((unsigned)rows), dim3(threads), 0, st, z, z_ld, coef, (B*)out, o_ld, n, eps));
    dlti_count_launch();
    return 0;
  }
  const size_t smem = (size_t)n * 4;
  if (smem > 47 * 1024) { dlti_set_error("poly_norm: rows of up to 12032 elements"); return DLTI_ERR_TOO_LARGE; }
  if (acc) {
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, poly_norm_kernel<__nv_bfloat16, true>, dim3((unsigned)rows), dim3(256), smem, st, z, z_ld, coef,
                                    (__nv_bfloat16*)out, o_ld, n, eps));
  } else {
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, poly_norm_kernel<T, false>, dim3((unsigned)rows), dim3(256), smem, st, z, z_ld, coef,
                                                      (T*)out, o_ld, n, eps)));
  }
  dlti_count_launch();
  return 0;
}

// n and split multiples of 8
DLTI_API int dlti_split_rows(float* acc, void* out, long long o_ld, float* tail, long long t_ld, long long rows, int n, int split, int dtype,
                             cudaStream_t st) {
  if (rows <= 0) return 0;
  if (n % 8 || split % 8 || split > n || o_ld % 8 || t_ld % 8 || dtype != DLTI_BF16) return DLTI_ERR_BAD_ARG;
  DLTI_CUDA_CHECK(dlti_launch_pdl(rows, split_rows_kernel<__nv_bfloat16>, dim3(grid_for(rows * (n / 8), 256)), dim3(256), 0, st, acc,
                                  (__nv_bfloat16*)out, o_ld, tail, t_ld, rows, n, split));
  dlti_count_launch();
  return 0;
}

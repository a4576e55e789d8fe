// Linear recurrences with an outer-product update, one state matrix per head:
//     S_t = a_t S_(t-1) + k_t (s_t v_t)^T,      o_t = S_t^T q_t + D v_t        (S is N x P, fp32)
// Mamba-2:    k = B, q = C (shared by the heads of a group), v = x, s_t = dt, a_t = exp(-exp(A_log) dt), D per head
// lightning:  a_t = one constant per head, s_t = 1, D = 0, silu on q, k, v as they are loaded
// mLSTM:      a_t = exp(f_t + m_(t-1) - m_t), s_t = exp(i_t - m_t) with log gates i_t, f_t and the running maximum
//             m_t = max(f_t + m_(t-1), i_t), m_0 = 0; n_t = a_t n_(t-1) + s_t k_t and o_t is divided by
//             max(|n_t . q_t|, exp(-m_t)) + 1e-6. n and m are state too; every slice of 32 columns of P, which is a CTA of
//             its own, keeps them for itself: vec [slots, heads, slices, N + 1] = n, then m.
// States live in slots [slots, heads, N, P] and are carried from step to step; a sequence whose step starts at position
// 0 starts from zero whatever its slot holds.
#include "recurrent.cuh"
#include "mma_sync.cuh"

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
  // mLSTM: raw gates [rows, >= 2 heads] fp32 (input gates, then forget gates), biases in the same order, soft cap, factor on q
  const float *gates, *gate_b; long long g_ld;
  float cap, q_scale;
  float* vec;
};

// log gates of an mLSTM head: cap tanh(z / cap), for the forget gate the logarithm of its sigmoid
__device__ __forceinline__ float log_in_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) { return -softplus_f(-cap * tanhf(z / cap)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

// Token-by-token form. CTA = (32 columns of P, head, sequence), 8 warps: lane = column, a warp owns the NR consecutive
// rows [warp * NR, ...), so q and k are warp-uniform shared-memory reads. TT tokens are staged at a time; the warps'
// partial outputs are summed once per stage.
constexpr int TT = 8;
template <typename T, int NR, bool ML>
__global__ void __launch_bounds__(256) scan_kernel(const ScanParams p, int slices, int conv_parts) {
  griddep_wait();
  griddep_launch();
  const int s = p.seq0 + blockIdx.z;
  if ((int)blockIdx.x >= slices) {
    if (blockIdx.y == 0) conv_tail<T>(p, s, blockIdx.x - slices, conv_parts);
    return;
  }
  __shared__ float sk[TT][8 * NR], sq[TT][8 * NR], sv[TT][32], part[TT][8][32], sstep[TT], sdecay[TT];
  __shared__ float nq[TT][8], floor_s[TT];                 // mLSTM: the warps' parts of n . q; exp(-m)
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
  constexpr int NV = (NR + 31) / 32;                       // entries of n per lane
  float nv[NV], m = 0.f;
  float* vec = ML ? p.vec + (((long long)(slot < 0 ? 0 : slot) * p.heads + h) * slices + blockIdx.x) * (p.N + 1) : nullptr;
  if constexpr (ML) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int r = warp * NR + lane + 32 * i;
      nv[i] = (slot >= 0 && start > 0 && lane + 32 * i < NR && r < p.N) ? vec[r] : 0.f;
    }
    if (slot >= 0 && start > 0) m = vec[p.N];
  }
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
      if (ML) {
        if (lane < 2) {
          const float z = p.gates[row * p.g_ld + lane * p.heads + h] + p.gate_b[lane * p.heads + h];
          if (lane == 0) sstep[warp] = log_in_gate(z, p.cap);
          else sdecay[warp] = log_forget_gate(z, p.cap);
        }
      } else if (lane == 0) {
        if (p.decay) {
          sstep[warp] = 1.f;
          sdecay[warp] = cdec;
        } else {
          const float step = softplus_f(Cvt<T>::to_f(reinterpret_cast<const T*>(p.dt)[row * p.dt_ld + h]) + p.dt_bias[h]);
          sstep[warp] = step;
          sdecay[warp] = decay_of(-expf(p.A_log[h]) * step);
        }
      }
    }
    __syncthreads();
    if constexpr (ML) {
      if (threadIdx.x == 0)                                // log gates -> factors, one token after the other
        for (int t = 0; t < nt; ++t) {
          const float f = sdecay[t] + m, i = sstep[t];
          m = fmaxf(f, i);
          sdecay[t] = decay_of(f - m);
          sstep[t] = expf(i - m);
          floor_s[t] = expf(-m);
        }
      __syncthreads();
    }
    for (int t = 0; t < nt; ++t) {
      const float a = sdecay[t];
      const float vv = sv[t][lane] * sstep[t];
      float acc = 0.f;
      if constexpr (ML) {
        float d = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (lane + 32 * i < NR) {
            nv[i] = fmaf(a, nv[i], sstep[t] * sk[t][warp * NR + lane + 32 * i]);
            d = fmaf(sq[t][warp * NR + lane + 32 * i], nv[i], d);
          }
        d = warp_sum(d);
        if (lane == 0) nq[t][warp] = d;
      }
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
      if constexpr (ML) {
        float d = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) d += nq[warp][w];
        o = o * p.q_scale / (fmaxf(fabsf(d * p.q_scale), floor_s[warp]) + 1e-6f);
      }
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
  if constexpr (ML) {
    if (slot >= 0) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int r = warp * NR + lane + 32 * i;
        if (lane + 32 * i < NR && r < p.N) vec[r] = nv[i];
      }
      if (threadIdx.x == 0) vec[p.N] = m;
    }
  }
}

template <typename T, bool ML>
int launch_scan(const ScanParams& p, int nseq, cudaStream_t st) {
  const int slices = (p.P + 31) / 32;
  const int conv_parts = p.conv_state ? (p.conv_C + 2047) / 2048 : 0;
  const dim3 grid(slices + conv_parts, p.heads, nseq);
  const long long rows = p.nd;                 // a programmatic dependent launch only pays in decode-sized steps
#define SCAN_CASE(NR)                                                                                                         \
  if (p.N <= 8 * NR) {                                                                                                        \
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows > 0 && p.seq0 + nseq <= p.nd ? rows : 1 << 20, scan_kernel<T, NR, ML>, grid, dim3(256), 0, st, \
                                    p, slices, conv_parts));                                                                  \
    dlti_count_launch();                                                                                                      \
    return 0;                                                                                                                 \
  }
  SCAN_CASE(4) SCAN_CASE(8) SCAN_CASE(16) SCAN_CASE(32) SCAN_CASE(64)
#undef SCAN_CASE
  dlti_set_error("linear_scan: states of up to 512 rows");
  return DLTI_ERR_TOO_LARGE;
}

// Chunked form for prompts, bf16: CTA = (32 columns of P, head, sequence), 64 tokens a chunk. With L_t the running sum of
// log2 a within the chunk and d_s = step size,
//     o_t   = 2^(L_t) S^T q_t + sum_(s <= t) [2^(L_t - L_s) d_s (k_s . q_t)] v_s
//     S'    = 2^(L_63) S + sum_s k_s [2^(L_63 - L_s) d_s v_s]^T
// q, k, v are exact bf16 operands; the three fp32 operands (S, the bracketed weights, the bracketed values) enter the
// tensor-core products as hi + lo bf16 pairs, so the recurrence keeps 16+ mantissa bits everywhere.
// Warps 0-3 compute the outputs (16 tokens each) from the S operand in shared memory; warps 4-7 meanwhile advance S, which
// lives in their fp32 accumulators (NT / 4 rows each), and publish it as the next operand once warps 0-3 have read the old
// one. Warp 4 also prepares the next chunk's decay vectors. One CTA-wide barrier per chunk.
//
// mLSTM: with F_t the running sum of log2 forget gates, a_s = log2 i_s - F_s and A_t = max(m, a_0 ... a_t) (m: the running
// maximum before the chunk, in log2) the maximum after token t is F_t + A_t, so the weight of s in t is 2^(a_s - A_t), that
// of the old state 2^(m - A_t): the same products with -A in the place of L and 2^a in that of the step sizes. n is one more
// column of the state product (its operand: the scaling factors themselves, hi in column 0 and lo in column 1), and
// n . q the row sums of the bracketed weights plus one more column of S^T q.
constexpr int CQ = 64, CP = 32, CPP = CP + 8;
template <int NT>
struct ChunkSmem {
  static constexpr int NP = NT + 8;
  static constexpr int QK = CQ * NP * 2, V = CQ * CPP * 2, STAGE = 2 * QK + V;          // bytes
  static constexpr int W = 2 * STAGE, S = W + 2 * V, VEC = S + 2 * NT * CPP * 2, VECS = 6 * CQ, NB = VEC + 2 * VECS * 4;
  static constexpr int BYTES = NB, BYTES_ML = NB + 2 * NT * 2;     // mLSTM: n as hi, lo
};
struct ChunkVec {                                                // one chunk's vectors, 64 each
  float *L, *step, *E, *F;                                       // L; d; 2^(L_63 - L_s) d; 2^(L_e - L_s) d, e = end of s's 16-block
  float *floor, *m;                                              // mLSTM: exp(-m_t); m before the chunk. L = -A, step = a
};
template <int NT, bool ML>
__global__ void __launch_bounds__(256, NT <= 128 ? 2 : 1) scan_chunk_kernel(const ScanParams p, int slices, int conv_parts) {
  using L = ChunkSmem<NT>;
  using bf16 = __nv_bfloat16;
  const int s = p.seq0 + blockIdx.z;
  if ((int)blockIdx.x >= slices) {
    if (blockIdx.y == 0) conv_tail<bf16>(p, s, blockIdx.x - slices, conv_parts);
    return;
  }
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  long long row0;
  int n, start;
  seq_rows(p, s, row0, n, start);
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = blockIdx.x * CP, ncol = min(CP, p.P - c0), grp = h / p.rep;
  const int slot = p.sslot[s];
  const bf16* q = reinterpret_cast<const bf16*>(p.q) + row0 * p.q_ld + (long long)grp * p.N;
  const bf16* k = reinterpret_cast<const bf16*>(p.k) + row0 * p.k_ld + (long long)grp * p.N;
  const bf16* v = reinterpret_cast<const bf16*>(p.v) + row0 * p.v_ld + (long long)h * p.P + c0;
  const float Dh = p.D ? p.D[h] : 0.f;
  auto vec = [&](int i) {
    float* f = reinterpret_cast<float*>(smem + L::VEC) + (i & 1) * L::VECS;
    return ChunkVec{f, f + CQ, f + 2 * CQ, f + 3 * CQ, f + 4 * CQ, f + 5 * CQ};
  };
  auto load = [&](int stage, int t0) {
    constexpr int STEP = 256 / (NT / 8);                         // rows per pass
    const uint32_t base = sb + stage * L::STAGE;
    const int r0 = threadIdx.x / (NT / 8), c = threadIdx.x % (NT / 8);
    const bool cok = c * 8 < p.N;
    const bf16* qp = q + (t0 + r0) * p.q_ld + c * 8;             // never dereferenced where a row or column is out of range
    const bf16* kp = k + (t0 + r0) * p.k_ld + c * 8;
    const uint32_t dst = base + (r0 * L::NP + c * 8) * 2;
#pragma unroll
    for (int i = 0; i < CQ / STEP; ++i) {
      const bool ok = cok && t0 + r0 + i * STEP < n;
      cp_async16(dst + i * STEP * L::NP * 2, ok ? qp : q, ok);
      cp_async16(dst + i * STEP * L::NP * 2 + L::QK, ok ? kp : k, ok);
      qp += STEP * p.q_ld;
      kp += STEP * p.k_ld;
    }
    const int r = threadIdx.x / (CP / 8), cv = threadIdx.x % (CP / 8);     // 64 rows x 4 pieces
    const bool ok = t0 + r < n && cv * 8 < ncol;
    cp_async16(base + 2 * L::QK + (r * CPP + cv * 8) * 2, ok ? v + (t0 + r) * p.v_ld + cv * 8 : v, ok);
    cp_async_commit();
  };
  load(0, 0);

  if (warp < 4) {
    // ---- outputs of 16 tokens per chunk ----
    const int scol = (lane & 3) * 2, tr = warp * 16 + (lane >> 2);
    int it = 0;
    for (int t0 = 0; t0 < n; t0 += CQ, ++it) {
      cp_async_wait<0>();
      __syncthreads();                                           // tile, vectors and S operand of this chunk are there
      if (t0 + CQ < n) load((it + 1) & 1, t0 + CQ);
      const uint32_t base = sb + (it & 1) * L::STAGE;
      const ChunkVec cv = vec(it);
      uint32_t qf[NT / 16][4];
      {
        const uint32_t qa = base + ((warp * 16 + (lane & 15)) * L::NP + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < NT / 16; ++kk) ldsm4(qf[kk], qa + kk * 32);
      }
      float o[CP / 8][4];
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) o[j][x] = 0.f;
      {
        const uint32_t sa = sb + L::S + ((lane & 15) * CPP + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < NT / 16; ++kk)
#pragma unroll
          for (int x = 0; x < 2; ++x)                            // hi, lo
#pragma unroll
            for (int j = 0; j < CP / 16; ++j) {
              uint32_t b[4];
              ldsm4_t(b, sa + x * (NT * CPP * 2) + (kk * 16 * CPP + j * 16) * 2);
              mma_bf16(o[2 * j], qf[kk], b[0], b[1]);
              mma_bf16(o[2 * j + 1], qf[kk], b[2], b[3]);
            }
      }
      float nq[4] = {};                                          // mLSTM: columns 0 and 1 (lanes 4 r): n . q, hi and lo part of n
      if constexpr (ML) {
        const uint8_t* nb = smem + L::NB + ((lane >> 2) & 1) * (NT * 2) + scol * 2;
#pragma unroll
        for (int kk = 0; kk < NT / 16; ++kk) {
          uint32_t b0 = *reinterpret_cast<const uint32_t*>(nb + kk * 32), b1 = *reinterpret_cast<const uint32_t*>(nb + kk * 32 + 16);
          if (lane >= 8) b0 = b1 = 0;
          mma_bf16(nq, qf[kk], b0, b1);
        }
      }
      asm volatile("bar.arrive 2, 256;" ::: "memory");           // the old S operand has been read
      const float lt[2] = {cv.L[tr], cv.L[tr + 8]};
      const float m0 = ML ? *cv.m : 0.f;
      const float el[2] = {ex2(lt[0] + m0), ex2(lt[1] + m0)};
      float rs[2] = {0.f, 0.f};                                  // mLSTM: row sums of the weights
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) o[j][x] *= el[x >> 1];
      for (int kb = 0; kb <= warp; ++kb) {                       // 16 keys at a time up to the diagonal
        float g0[4] = {}, g1[4] = {};
        const uint32_t ka = base + L::QK + ((kb * 16 + (lane & 7) + ((lane >> 4) << 3)) * L::NP + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < NT / 16; ++kk) {
          uint32_t b[4];
          ldsm4(b, ka + kk * 32);
          mma_bf16(g0, qf[kk], b[0], b[1]);
          mma_bf16(g1, qf[kk], b[2], b[3]);
        }
        if (kb < warp) {                                         // all keys precede all tokens: factored through the block's end
          const float le = cv.L[kb * 16 + 15];
          const float f0 = ex2(lt[0] - le), f1 = ex2(lt[1] - le);
          const float2 a = *reinterpret_cast<const float2*>(cv.F + kb * 16 + scol), b = *reinterpret_cast<const float2*>(cv.F + kb * 16 + 8 + scol);
          g0[0] *= a.x * f0; g0[1] *= a.y * f0; g0[2] *= a.x * f1; g0[3] *= a.y * f1;
          g1[0] *= b.x * f0; g1[1] *= b.y * f0; g1[2] *= b.x * f1; g1[3] *= b.y * f1;
        } else {
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int t = tr + 8 * (x >> 1);
            const int u0 = kb * 16 + scol + (x & 1), u1 = u0 + 8;
            if constexpr (ML) {
              g0[x] = u0 <= t ? g0[x] * ex2(lt[x >> 1] + cv.step[u0]) : 0.f;
              g1[x] = u1 <= t ? g1[x] * ex2(lt[x >> 1] + cv.step[u1]) : 0.f;
            } else {
              g0[x] = u0 <= t ? g0[x] * cv.step[u0] * ex2(lt[x >> 1] - cv.L[u0]) : 0.f;
              g1[x] = u1 <= t ? g1[x] * cv.step[u1] * ex2(lt[x >> 1] - cv.L[u1]) : 0.f;
            }
          }
        }
        if constexpr (ML) {
#pragma unroll
          for (int x = 0; x < 4; ++x) rs[x >> 1] += g0[x] + g1[x];
        }
        uint32_t hi[4], lo[4];
        split_pair(g0[0], g0[1], hi[0], lo[0]);
        split_pair(g0[2], g0[3], hi[1], lo[1]);
        split_pair(g1[0], g1[1], hi[2], lo[2]);
        split_pair(g1[2], g1[3], hi[3], lo[3]);
        const uint32_t va = base + 2 * L::QK + ((kb * 16 + (lane & 15)) * CPP + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int j = 0; j < CP / 16; ++j) {
          uint32_t b[4];
          ldsm4_t(b, va + j * 32);
          mma_bf16(o[2 * j], hi, b[0], b[1]);
          mma_bf16(o[2 * j + 1], hi, b[2], b[3]);
          mma_bf16(o[2 * j], lo, b[0], b[1]);
          mma_bf16(o[2 * j + 1], lo, b[2], b[3]);
        }
      }
      const bf16* sv = reinterpret_cast<const bf16*>(smem + (it & 1) * L::STAGE + 2 * L::QK);
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int t = tr + 8 * y;
        float f = 1.f;
        if constexpr (ML) {
          rs[y] += __shfl_xor_sync(0xffffffffu, rs[y], 1);
          rs[y] += __shfl_xor_sync(0xffffffffu, rs[y], 2);
          const float old = __shfl_sync(0xffffffffu, nq[2 * y] + nq[2 * y + 1], lane & ~3);
          f = p.q_scale / (fmaxf(fabsf(p.q_scale * (el[y] * old + rs[y])), cv.floor[t]) + 1e-6f);
        }
        if (t0 + t < n) {
          bf16* orow = reinterpret_cast<bf16*>(p.out) + (row0 + t0 + t) * p.o_ld + (long long)h * p.P + c0;
#pragma unroll
          for (int j = 0; j < CP / 8; ++j) {
            const int c = j * 8 + scol;
            if (c >= ncol) continue;
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + t * CPP + c));
            if constexpr (ML) *reinterpret_cast<__nv_bfloat162*>(orow + c) = __floats2bfloat162_rn(o[j][2 * y] * f, o[j][2 * y + 1] * f);
            else *reinterpret_cast<__nv_bfloat162*>(orow + c) = __floats2bfloat162_rn(o[j][2 * y] + Dh * x.x, o[j][2 * y + 1] + Dh * x.y);
          }
        }
      }
    }
    return;
  }

  // ---- state ----
  const int sw = warp - 4;
  constexpr float LOG2E = 1.4426950408889634f;
  const float eA = ML || p.decay ? 0.f : expf(p.A_log[h]) * LOG2E;
  const float la_c = !ML && p.decay ? fmaxf(logf(p.decay[h]), -80.f) * LOG2E : 0.f;
  const float bias = ML ? p.gate_b[h] : (p.decay ? 0.f : p.dt_bias[h]);
  const float bias_f = ML ? p.gate_b[p.heads + h] : 0.f;
  float* vecs = ML ? p.vec + (((long long)(slot < 0 ? 0 : slot) * p.heads + h) * slices + blockIdx.x) * (p.N + 1) : nullptr;
  float m = 0.f;                                                 // warp 4, mLSTM: log2 of the running maximum
  // warp 4: step sizes and decays of the chunk at t0, two consecutive tokens a lane
  auto raw_dt = [&](int t0, float (&d)[4]) {                     // mLSTM: input gates, then forget gates
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int t = t0 + 2 * lane + y;
      if constexpr (ML) {
        d[y] = t < n ? p.gates[(row0 + t) * p.g_ld + h] + bias : 0.f;
        d[2 + y] = t < n ? p.gates[(row0 + t) * p.g_ld + p.heads + h] + bias_f : 0.f;
      } else
      d[y] = (!p.decay && t < n) ? __bfloat162float(reinterpret_cast<const bf16*>(p.dt)[(row0 + t) * p.dt_ld + h]) + bias : 0.f;
    }
  };
  auto prepare_ml = [&](int i, int t0, const float (&d)[4]) {
    float f[2], a[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) f[y] = t0 + 2 * lane + y < n ? log_forget_gate(d[2 + y], p.cap) * LOG2E : 0.f;
    f[1] += f[0];
    float x = f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x += y;
    }
    const float F1 = x, F0 = x - f[1] + f[0];
#pragma unroll
    for (int y = 0; y < 2; ++y) a[y] = t0 + 2 * lane + y < n ? log_in_gate(d[y], p.cap) * LOG2E - (y ? F1 : F0) : -INFINITY;
    x = fmaxf(a[0], a[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x = fmaxf(x, y);
    }
    float before = __shfl_up_sync(0xffffffffu, x, 1);
    before = lane == 0 ? m : fmaxf(m, before);
    const float A0 = fmaxf(before, a[0]), A1 = fmaxf(A0, a[1]);
    const float last = __shfl_sync(0xffffffffu, A1, 31), Ae = __shfl_sync(0xffffffffu, A1, lane | 7);
    const ChunkVec cv = vec(i);
    *reinterpret_cast<float2*>(cv.L + 2 * lane) = make_float2(-A0, -A1);
    *reinterpret_cast<float2*>(cv.step + 2 * lane) = make_float2(a[0], a[1]);
    *reinterpret_cast<float2*>(cv.E + 2 * lane) = make_float2(ex2(a[0] - last), ex2(a[1] - last));
    *reinterpret_cast<float2*>(cv.F + 2 * lane) = make_float2(ex2(a[0] - Ae), ex2(a[1] - Ae));
    *reinterpret_cast<float2*>(cv.floor + 2 * lane) = make_float2(ex2(-(F0 + A0)), ex2(-(F1 + A1)));
    if (lane == 0) *cv.m = m;
    m = __shfl_sync(0xffffffffu, F1, 31) + last;
  };
  auto prepare = [&](int i, int t0, const float (&d)[4]) {
    float step[2], l[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const bool ok = t0 + 2 * lane + y < n;
      step[y] = !ok ? 0.f : (p.decay ? 1.f : softplus_f(d[y]));
      l[y] = !ok ? 0.f : (p.decay ? la_c : -eA * step[y]);
    }
    l[1] += l[0];
    float x = l[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x += y;
    }
    const float before = x - l[1];
    const float total = __shfl_sync(0xffffffffu, x, 31);
    const float le = __shfl_sync(0xffffffffu, x, lane | 7);      // end of this 16-token block
    const float l0 = before + l[0], l1 = x;
    const ChunkVec cv = vec(i);
    *reinterpret_cast<float2*>(cv.L + 2 * lane) = make_float2(l0, l1);
    *reinterpret_cast<float2*>(cv.step + 2 * lane) = make_float2(step[0], step[1]);
    *reinterpret_cast<float2*>(cv.E + 2 * lane) = make_float2(ex2(total - l0) * step[0], ex2(total - l1) * step[1]);
    *reinterpret_cast<float2*>(cv.F + 2 * lane) = make_float2(ex2(le - l0) * step[0], ex2(le - l1) * step[1]);
  };
  constexpr int MT = NT / 64;                                    // 16-row state tiles of a warp
  float S[MT][CP / 8][4];
  float* st = p.state + (((long long)(slot < 0 ? 0 : slot) * p.heads + h) * p.N) * p.P + c0;
  const int srow = sw * (NT / 4) + (lane >> 2), scol = (lane & 3) * 2;
  const bool have = slot >= 0 && start > 0;
  float ns[ML ? MT : 1][4];                                      // mLSTM: columns 0 (from hi) and 1 (from lo) in lanes 4 r; n is their sum
  auto publish = [&]() {                                         // S as hi / lo operands
    if constexpr (ML) {
      if ((lane & 3) == 0)
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            const float x = ns[i][2 * y] + ns[i][2 * y + 1];
            const bf16 hi = __float2bfloat16(x);
            bf16* nb = reinterpret_cast<bf16*>(smem + L::NB) + srow + i * 16 + 8 * y;
            nb[0] = hi;
            nb[NT] = __float2bfloat16(x - __bfloat162float(hi));
          }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          uint32_t hi, lo;
          split_pair(S[i][j][2 * y], S[i][j][2 * y + 1], hi, lo);
          const int off = ((srow + i * 16 + 8 * y) * CPP + j * 8 + scol) * 2;
          *reinterpret_cast<uint32_t*>(smem + L::S + off) = hi;
          *reinterpret_cast<uint32_t*>(smem + L::S + NT * CPP * 2 + off) = lo;
        }
  };
  float d[4] = {0.f, 0.f, 0.f, 0.f};
  if constexpr (ML) {
    if (have) m = vecs[p.N] * LOG2E;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int r = srow + i * 16 + 8 * y;
        ns[i][2 * y] = have && (lane & 3) == 0 && r < p.N ? vecs[r] : 0.f;
        ns[i][2 * y + 1] = 0.f;
      }
  }
  if (sw == 0) {
    raw_dt(0, d);
    if constexpr (ML) prepare_ml(0, 0, d);
    else prepare(0, 0, d);
    raw_dt(CQ, d);
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int r = srow + i * 16 + 8 * y, c = j * 8 + scol;
        const bool ok = have && r < p.N && c < ncol;             // ncol is a multiple of 8
        S[i][j][2 * y] = ok ? st[(long long)r * p.P + c] : 0.f;
        S[i][j][2 * y + 1] = ok ? st[(long long)r * p.P + c + 1] : 0.f;
      }
  publish();
  int it = 0;
  for (int t0 = 0; t0 < n; t0 += CQ, ++it) {
    cp_async_wait<0>();
    __syncthreads();
    if (t0 + CQ < n) load((it + 1) & 1, t0 + CQ);
    const uint32_t base = sb + (it & 1) * L::STAGE;
    const ChunkVec cv = vec(it);
    const bf16* sv = reinterpret_cast<const bf16*>(smem + (it & 1) * L::STAGE + 2 * L::QK);
#pragma unroll
    for (int i = 0; i < CQ * CP / 2 / 128; ++i) {                // scaled values as hi / lo operands
      const int r = (threadIdx.x - 128) / (CP / 2) + i * (128 / (CP / 2)), c = 2 * (threadIdx.x % (CP / 2));
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + r * CPP + c));
      const float e = cv.E[r];
      uint32_t hi, lo;
      split_pair(x.x * e, x.y * e, hi, lo);
      *reinterpret_cast<uint32_t*>(smem + L::W + (r * CPP + c) * 2) = hi;
      *reinterpret_cast<uint32_t*>(smem + L::W + L::V + (r * CPP + c) * 2) = lo;
    }
    const float keep = ex2(cv.L[CQ - 1] + (ML ? *cv.m : 0.f));
#pragma unroll
    for (int i = 0; i < MT; ++i) {
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) S[i][j][x] *= keep;
      if constexpr (ML)
#pragma unroll
        for (int x = 0; x < 4; ++x) ns[i][x] *= keep;
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");               // scaled values written (warps 4-7)
#pragma unroll
    for (int kb = 0; kb < CQ / 16; ++kb) {
      uint32_t w[2][CP / 16][4];
      const uint32_t wa = sb + L::W + ((kb * 16 + (lane & 15)) * CPP + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int j = 0; j < CP / 16; ++j) ldsm4_t(w[x][j], wa + x * L::V + j * 32);
      uint32_t e0 = 0, e1 = 0;                                   // mLSTM: factors of keys 16 kb .. as columns 0 (hi) and 1 (lo)
      if constexpr (ML) {
        const float2 u = *reinterpret_cast<const float2*>(cv.E + kb * 16 + scol), v2 = *reinterpret_cast<const float2*>(cv.E + kb * 16 + 8 + scol);
        uint32_t lo0, lo1;
        split_pair(u.x, u.y, e0, lo0);
        split_pair(v2.x, v2.y, e1, lo1);
        if (lane >= 4) { e0 = lane < 8 ? lo0 : 0; e1 = lane < 8 ? lo1 : 0; }
      }
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        // A = K^T: rows n, columns s, read transposed from K [s][n]
        uint32_t a[4];
        ldsm4_t(a, base + L::QK + ((kb * 16 + (lane & 7) + ((lane >> 4) << 3)) * L::NP + sw * (NT / 4) + i * 16 + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
          for (int j = 0; j < CP / 16; ++j) {
            mma_bf16(S[i][2 * j], a, w[x][j][0], w[x][j][1]);
            mma_bf16(S[i][2 * j + 1], a, w[x][j][2], w[x][j][3]);
          }
        if constexpr (ML) mma_bf16(ns[i], a, e0, e1);
      }
    }
    if (sw == 0 && t0 + CQ < n) {
      if constexpr (ML) prepare_ml(it + 1, t0 + CQ, d);
      else prepare(it + 1, t0 + CQ, d);
      raw_dt(t0 + 2 * CQ, d);
    }
    asm volatile("bar.sync 2, 256;" ::: "memory");               // warps 0-3 have read the old operand
    publish();
  }
  if (slot >= 0) {
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int r = srow + i * 16 + 8 * y, c = j * 8 + scol;
          if (r < p.N && c < ncol) {
            st[(long long)r * p.P + c] = S[i][j][2 * y];
            st[(long long)r * p.P + c + 1] = S[i][j][2 * y + 1];
          }
        }
    if constexpr (ML) {
      if ((lane & 3) == 0)
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            const int r = srow + i * 16 + 8 * y;
            if (r < p.N) vecs[r] = ns[i][2 * y] + ns[i][2 * y + 1];
          }
      if (sw == 0 && lane == 0) vecs[p.N] = m * (1.f / LOG2E);
    }
  }
}

template <int NT, bool ML>
int launch_chunk(const ScanParams& p, int nseq, cudaStream_t st) {
  static bool done[64] = {};
  const int bytes = ML ? ChunkSmem<NT>::BYTES_ML : ChunkSmem<NT>::BYTES;
  int dev = 0;
  DLTI_CUDA_CHECK(cudaGetDevice(&dev));
  if (!done[dev & 63]) {
    DLTI_CUDA_CHECK(cudaFuncSetAttribute(scan_chunk_kernel<NT, ML>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    done[dev & 63] = true;
  }
  const int slices = (p.P + CP - 1) / CP;
  const int conv_parts = p.conv_state ? (p.conv_C + 2047) / 2048 : 0;
  scan_chunk_kernel<NT, ML><<<dim3(slices + conv_parts, p.heads, nseq), 256, bytes, st>>>(p, slices, conv_parts);
  dlti_count_launch();
  return (int)cudaGetLastError();
}

// x = silu(x) in place, rounded to T
template <typename T>
__global__ void silu_rows_kernel(T* __restrict__ x, long long ld, long long rows, int n) {
  const int vec = n >> 3;
  const long long total = rows * vec;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / vec;
    int4* p = reinterpret_cast<int4*>(x + t * ld) + (int)(i - t * vec);
    int4 v = *p;
    uint32_t* u = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = Cvt<T>::unpack2(u[j]);
      u[j] = Cvt<T>::pack2(f.x / (1.f + __expf(-f.x)), f.y / (1.f + __expf(-f.y)));
    }
    *p = v;
  }
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
  if (dtype == DLTI_BF16) return launch_scan<__nv_bfloat16, false>(p, nseq, st);
  if (dtype == DLTI_FP32) return launch_scan<float, false>(p, nseq, st);
  return DLTI_ERR_UNSUPPORTED;
}

// The chunked tensor-core form of the same for prompt sequences: bf16, N and P multiples of 8, N <= 256, q / k / v rows
// 16-byte aligned, no silu (see dlti_silu_rows).
DLTI_API int dlti_linear_scan_chunked(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, int rep,
                                      const float* decay, const void* dt, long long dt_ld, const float* dt_bias, const float* A_log,
                                      const float* D, float* state, const int* sslot, const int* ctx, const int* cu, int nd, int seq0,
                                      int nseq, int heads, int N, int P, void* out, long long o_ld, const void* conv_src,
                                      long long conv_ld, int conv_col, int conv_rows, int conv_C, void* conv_state, cudaStream_t st) {
  if (nseq <= 0) return 0;
  if (heads < 1 || rep < 1 || nseq > 65535 || (!decay && (!dt || !dt_bias || !A_log))) return DLTI_ERR_BAD_ARG;
  if (N % 8 || P % 8 || q_ld % 8 || k_ld % 8 || v_ld % 8 || o_ld % 2 ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15)) {
    dlti_set_error("linear_scan_chunked: 16-byte aligned rows, N and P multiples of 8");
    return DLTI_ERR_BAD_ARG;
  }
  if (conv_rows <= 0) conv_state = nullptr;
  ScanParams p{q, k, v, q_ld, k_ld, v_ld, rep, 0, decay, dt, dt_ld, dt_bias, A_log, D, state, sslot, ctx, cu,
               nd, seq0, heads, N, P, out, o_ld, conv_src, conv_ld, conv_col, conv_rows, conv_C, conv_state};
  if (N <= 64) return launch_chunk<64, false>(p, nseq, st);
  if (N <= 128) return launch_chunk<128, false>(p, nseq, st);
  if (N <= 256) return launch_chunk<256, false>(p, nseq, st);
  dlti_set_error("linear_scan_chunked: states of up to 256 rows");
  return DLTI_ERR_TOO_LARGE;
}

// mLSTM over the sequences [seq0, seq0 + nseq): q, k rows heads * N, v rows heads * P wide; gates / gate_b: see ScanParams; state
// [slots, heads, N, P], vec [slots, heads, ceil(P / 32), N + 1]. chunked: the tensor-core form (bf16, N and P multiples of 8,
// N <= 256, 16-byte aligned rows), else token by token (N <= 512).
DLTI_API int dlti_mlstm_scan(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, const float* gates,
                             long long g_ld, const float* gate_b, float cap, float q_scale, float* state, float* vec, const int* sslot,
                             const int* ctx, const int* cu, int nd, int seq0, int nseq, int heads, int N, int P, void* out, long long o_ld,
                             int chunked, int dtype, cudaStream_t st) {
  if (nseq <= 0) return 0;
  if (heads < 1 || N < 1 || P < 1 || nseq > 65535 || !gates || !gate_b || !(cap > 0.f)) return DLTI_ERR_BAD_ARG;
  ScanParams p{};
  p.q = q; p.k = k; p.v = v; p.q_ld = q_ld; p.k_ld = k_ld; p.v_ld = v_ld; p.rep = 1;
  p.gates = gates; p.g_ld = g_ld; p.gate_b = gate_b; p.cap = cap; p.q_scale = q_scale; p.state = state; p.vec = vec;
  p.sslot = sslot; p.ctx = ctx; p.cu = cu; p.nd = nd; p.seq0 = seq0; p.heads = heads; p.N = N; p.P = P; p.out = out; p.o_ld = o_ld;
  if (!chunked) {
    if (dtype == DLTI_BF16) return launch_scan<__nv_bfloat16, true>(p, nseq, st);
    if (dtype == DLTI_FP32) return launch_scan<float, true>(p, nseq, st);
    return DLTI_ERR_UNSUPPORTED;
  }
  if (dtype != DLTI_BF16 || N % 8 || P % 8 || N > 256 || q_ld % 8 || k_ld % 8 || v_ld % 8 || o_ld % 2 ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15)) {
    dlti_set_error("mlstm_scan, chunked: bf16, 16-byte aligned rows, N and P multiples of 8, N <= 256");
    return DLTI_ERR_BAD_ARG;
  }
  if (N <= 64) return launch_chunk<64, true>(p, nseq, st);
  if (N <= 128) return launch_chunk<128, true>(p, nseq, st);
  return launch_chunk<256, true>(p, nseq, st);
}

DLTI_API int dlti_silu_rows(void* x, long long ld, long long rows, int n, int dtype, cudaStream_t st) {
  if (rows <= 0 || n <= 0) return 0;
  if (dtype != DLTI_BF16) return DLTI_ERR_UNSUPPORTED;
  if (n % 8 || ld % 8 || (reinterpret_cast<uintptr_t>(x) & 15)) return DLTI_ERR_BAD_ARG;
  const long long g = (rows * (n / 8) + 255) / 256, cap = (long long)dlti_num_sms() * 16;
  silu_rows_kernel<__nv_bfloat16><<<(unsigned)(g < cap ? g : cap), 256, 0, st>>>((__nv_bfloat16*)x, ld, rows, n);
  dlti_count_launch();
  return (int)cudaGetLastError();
}

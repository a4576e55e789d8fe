// Gated delta rule, one state matrix per head (S is N x P, fp32):
//     S <- g_t S,   u_t = b_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t
// with unit keys and queries (queries also times N^-1/2) shared by the heads of a group, g_t = exp(-exp(A_log) softplus(a_t +
// dt_bias)) and b_t the sigmoid of a projected number. States live in slots [slots, heads, N, P] and are carried from step to
// step; a sequence whose step starts at position 0 starts from zero whatever its slot holds.
//
//   delta_kernel        token by token: decode rows, short portions, fp32
//   delta_prep_kernel   prompts, everything of a chunk of 64 tokens that does not need the state: all chunks at once
//   delta_chunk_kernel  prompts, one chunk after the other with those results
#include "recurrent.cuh"
#include "mma_sync.cuh"

namespace {

constexpr float UNIT_EPS = 1e-6f;

struct DeltaParams {
  const void *q, *k, *v;
  long long q_ld, k_ld, v_ld;
  const float* gates; long long g_ld;      // [rows, >= 2 heads]: raw a, then raw b
  const float *A_log, *dt_bias;
  float* state;
  const int *sslot, *ctx, *cu;
  int nd, seq0, heads, rep, N, P;          // rep: heads per query/key head
  void* out; long long o_ld;
  const void* conv_src; long long conv_ld; int conv_col, conv_rows, conv_C;
  void* conv_state;
  uint8_t* ws;                             // chunked form: results of delta_prep_kernel
};

__device__ __forceinline__ float log_decay(const DeltaParams& p, long long row, int h) {
  return -expf(p.A_log[h]) * softplus_f(p.gates[row * p.g_ld + h] + p.dt_bias[h]);
}
__device__ __forceinline__ float step_share(const DeltaParams& p, long long row, int h) {
  return 1.f / (1.f + expf(-p.gates[row * p.g_ld + p.heads + h]));
}

// CTA = (32 columns of P, head, sequence), 8 warps: lane = column, a warp owns the NR consecutive rows [warp * NR, ...). With the
// old state's products k^T S and q^T S known, u and o = g q^T S + (k . q) u follow without a second pass, so a token costs one
// exchange between the warps. TT tokens are staged at a time.
constexpr int TT = 8;
template <typename T, int NR>
__global__ void __launch_bounds__(256) delta_kernel(const DeltaParams p, int slices, int conv_parts) {
  griddep_wait();
  griddep_launch();
  const int s = p.seq0 + blockIdx.z;
  if ((int)blockIdx.x >= slices) {
    if (blockIdx.y == 0) conv_tail<T>(p, s, blockIdx.x - slices, conv_parts);
    return;
  }
  __shared__ float sk[TT][8 * NR], sq[TT][8 * NR], sv[TT][32], sb[TT], sg[TT], skq[TT];
  __shared__ float2 part[2][8][32];
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
  const T* q = reinterpret_cast<const T*>(p.q) + (long long)grp * p.N;
  const T* k = reinterpret_cast<const T*>(p.k) + (long long)grp * p.N;
  const T* v = reinterpret_cast<const T*>(p.v) + (long long)h * p.P;
  const float q_scale = 1.f / sqrtf((float)p.N);
  for (int t0 = 0; t0 < n; t0 += TT) {
    const int nt = min(TT, n - t0);
    __syncthreads();
    if (warp < nt) {                                       // a warp prepares one token
      const long long row = row0 + t0 + warp;
      float kk = 0.f, qq = 0.f, kq = 0.f;
      for (int i = lane; i < 8 * NR; i += 32) {
        const float a = i < p.N ? Cvt<T>::to_f(k[row * p.k_ld + i]) : 0.f, b = i < p.N ? Cvt<T>::to_f(q[row * p.q_ld + i]) : 0.f;
        sk[warp][i] = a;
        sq[warp][i] = b;
        kk = fmaf(a, a, kk);
        qq = fmaf(b, b, qq);
        kq = fmaf(a, b, kq);
      }
      const float rk = 1.f / sqrtf(warp_sum(kk) + UNIT_EPS), rq = q_scale / sqrtf(warp_sum(qq) + UNIT_EPS);
      kq = warp_sum(kq);
      for (int i = lane; i < 8 * NR; i += 32) {
        sk[warp][i] *= rk;
        sq[warp][i] *= rq;
      }
      sv[warp][lane] = colok ? Cvt<T>::to_f(v[row * p.v_ld + col]) : 0.f;
      if (lane == 0) {
        skq[warp] = kq * rk * rq;
        sb[warp] = step_share(p, row, h);
        sg[warp] = decay_of(log_decay(p, row, h));
      }
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        a = fmaf(sk[t][warp * NR + i], S[i], a);
        b = fmaf(sq[t][warp * NR + i], S[i], b);
      }
      part[t & 1][warp][lane] = make_float2(a, b);
      __syncthreads();
      a = b = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const float2 x = part[t & 1][w][lane];
        a += x.x;
        b += x.y;
      }
      const float g = sg[t], u = sb[t] * (sv[t][lane] - g * a);
#pragma unroll
      for (int i = 0; i < NR; ++i) S[i] = fmaf(g, S[i], sk[t][warp * NR + i] * u);
      if (warp == t && colok)
        reinterpret_cast<T*>(p.out)[(row0 + t0 + t) * p.o_ld + (long long)h * p.P + col] = Cvt<T>::from_f(fmaf(skq[t], u, g * b));
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

// Chunks of 64 tokens. L_t: running sum of log2 g in the chunk, rk_t / rq_t: reciprocal lengths (rq with N^-1/2), S: the state
// before the chunk. The u of a chunk solve a unit lower triangular system:
//     u_t + sum_(s < t) A_ts u_s = b_t (v_t - 2^(L_t) rk_t S^T k_t) =: r_t,    A_ts = b_t 2^(L_t - L_s) rk_t rk_s (k_t . k_s)
//     o_t = 2^(L_t) rq_t S^T q_t + sum_(s <= t) M_ts u_s,                      M_ts = 2^(L_t - L_s) rq_t rk_s (q_t . k_s)
//     S'  = 2^(L_63) S + sum_s k_s (2^(L_63 - L_s) rk_s u_s)^T
// delta_prep_kernel leaves inverse(I + A) and M as hi / lo bf16 A-fragments of mma.m16n8k16 (block row w, block column kb <= w) and
// the vectors 2^(L_t) rk_t, 2^(L_t) rq_t, b_t, 2^(L_63 - L_t) rk_t, 2^(L_63). Raw keys, queries and values are exact bf16 operands;
// every fp32 operand enters its products as hi + lo.
constexpr int CQ = 64, CP = 32, CPP = CP + 8;
constexpr int FRAG_BYTES = 4 * 4 * 32 * 32;                // [row block][column block][lane][hi 16 bytes, lo 16 bytes]
constexpr int VEC_FLOATS = 4 * CQ + 4;
constexpr int WS_BYTES = 2 * FRAG_BYTES + VEC_FLOATS * 4 + 112;            // multiple of 128
static_assert(WS_BYTES % 128 == 0, "");
// chunks of the prompts before sequence i (an upper bound that needs no prefix sum), for rows counted from the first prompt row
__host__ __device__ __forceinline__ long long chunk_base(long long row, int i) { return row / CQ + i; }
__device__ __forceinline__ uint8_t* chunk_ws(const DeltaParams& p, long long row0, int s, int chunk, int h) {
  return p.ws + ((chunk_base(row0 - p.nd, s - p.nd) + chunk) * p.heads + h) * WS_BYTES;
}

template <int NT>
__device__ __forceinline__ void load_rows(uint32_t dst, const __nv_bfloat16* src, long long ld, int t0, int n, int N, int tid, int threads) {
  constexpr int NP = NT + 8, PR = NT / 8;
  for (int i = tid; i < CQ * PR; i += threads) {
    const int r = i / PR, c = i % PR;
    const bool ok = t0 + r < n && c * 8 < N;
    cp_async16(dst + (r * NP + c * 8) * 2, ok ? src + (long long)(t0 + r) * ld + c * 8 : src, ok);
  }
}

template <int NT>
struct PrepSmem {
  static constexpr int NP = NT + 8, QK = CQ * NP * 2, A = 2 * QK, AP = CQ + 4, VEC = A + CQ * AP * 4, BYTES = VEC + 5 * CQ * 4;
};
template <int NT>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaParams p) {
  using L = PrepSmem<NT>;
  using bf16 = __nv_bfloat16;
  extern __shared__ __align__(128) uint8_t smem[];
  const int s = p.seq0 + blockIdx.z, h = blockIdx.y, grp = h / p.rep;
  long long row0;
  int n, start;
  seq_rows(p, s, row0, n, start);
  const int t0 = blockIdx.x * CQ;
  if (t0 >= n) return;
  const uint32_t sb = smem_u32(smem);
  float* A = reinterpret_cast<float*>(smem + L::A);
  float *vL = reinterpret_cast<float*>(smem + L::VEC), *vb = vL + CQ, *rk = vb + CQ, *rq = rk + CQ;
  uint8_t* ws = chunk_ws(p, row0, s, blockIdx.x, h);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  load_rows<NT>(sb, reinterpret_cast<const bf16*>(p.k) + row0 * p.k_ld + (long long)grp * p.N, p.k_ld, t0, n, p.N, threadIdx.x, 256);
  load_rows<NT>(sb + L::QK, reinterpret_cast<const bf16*>(p.q) + row0 * p.q_ld + (long long)grp * p.N, p.q_ld, t0, n, p.N, threadIdx.x, 256);
  cp_async_commit();
  if (warp == 0) {                                         // two consecutive tokens a lane
    float l[2], b[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int t = t0 + 2 * lane + y;
      l[y] = t < n ? log_decay(p, row0 + t, h) * 1.4426950408889634f : 0.f;
      b[y] = t < n ? step_share(p, row0 + t, h) : 0.f;
    }
    l[1] += l[0];
    float x = l[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x += y;
    }
    vL[2 * lane] = x - l[1] + l[0];
    vL[2 * lane + 1] = x;
    vb[2 * lane] = b[0];
    vb[2 * lane + 1] = b[1];
  }
  cp_async_wait<0>();
  __syncthreads();
  {                                                        // lengths: four threads a row
    const int r = threadIdx.x >> 2, part = threadIdx.x & 3;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const uint4* row = reinterpret_cast<const uint4*>(smem + x * L::QK + r * L::NP * 2);
      float ss = 0.f;
      for (int c = part; c < NT / 8; c += 4) {
        const uint4 v = row[c];
        const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = Cvt<bf16>::unpack2(u[j]);
          ss += f.x * f.x + f.y * f.y;
        }
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (part == 0) (x ? rq : rk)[r] = (x ? 1.f / sqrtf((float)p.N) : 1.f) / sqrtf(ss + UNIT_EPS);
    }
  }
  __syncthreads();
  {                                                        // products with the keys: warps 0-3 of the keys, warps 4-7 of the queries
    const int w = warp & 3;
    const bool of_q = warp >= 4;
    const int tr = w * 16 + (lane >> 2), sc = (lane & 3) * 2;
    uint32_t f[NT / 16][4];
    const uint32_t fa = sb + (of_q ? L::QK : 0) + ((w * 16 + (lane & 15)) * L::NP + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int kk = 0; kk < NT / 16; ++kk) ldsm4(f[kk], fa + kk * 32);
    uint4* frag = reinterpret_cast<uint4*>(ws + FRAG_BYTES);
    float row_f[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) row_f[y] = of_q ? rq[tr + 8 * y] : vb[tr + 8 * y] * rk[tr + 8 * y];
    for (int kb = 0; kb < 4; ++kb) {
      float g[2][4] = {};
      if (kb <= w) {
        const uint32_t ka = sb + ((kb * 16 + (lane & 7) + ((lane >> 4) << 3)) * L::NP + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < NT / 16; ++kk) {
          uint32_t b[4];
          ldsm4(b, ka + kk * 32);
          mma_bf16(g[0], f[kk], b[0], b[1]);
          mma_bf16(g[1], f[kk], b[2], b[3]);
        }
#pragma unroll
        for (int z = 0; z < 2; ++z)
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int t = tr + 8 * (x >> 1), u = kb * 16 + z * 8 + sc + (x & 1);
            const bool seen = of_q ? u <= t : u < t;
            g[z][x] = seen ? g[z][x] * row_f[x >> 1] * rk[u] * ex2(vL[t] - vL[u]) : 0.f;
          }
      }
      if (of_q) {
        if (kb <= w) {
          uint32_t hi[4], lo[4];
          split_pair(g[0][0], g[0][1], hi[0], lo[0]);
          split_pair(g[0][2], g[0][3], hi[1], lo[1]);
          split_pair(g[1][0], g[1][1], hi[2], lo[2]);
          split_pair(g[1][2], g[1][3], hi[3], lo[3]);
          uint4* o = frag + ((w * 4 + kb) * 32 + lane) * 2;
          o[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          o[1] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      } else {
#pragma unroll
        for (int z = 0; z < 2; ++z)
#pragma unroll
          for (int y = 0; y < 2; ++y)
            *reinterpret_cast<float2*>(A + (tr + 8 * y) * L::AP + kb * 16 + z * 8 + sc) = make_float2(g[z][2 * y], g[z][2 * y + 1]);
      }
    }
  }
  __syncthreads();
  // The inverse I takes the place of the keys and queries. Its 16 x 16 blocks on the diagonal by forward substitution, a column a
  // thread; then one diagonal of blocks after the other: I_ij = -I_ii sum_(j <= k < i) A_ik I_kj, an element a thread.
  float* I = reinterpret_cast<float*>(smem);
  static_assert(2 * L::QK >= CQ * L::AP * 4, "");
  if (threadIdx.x < CQ) {
    const int b = threadIdx.x & ~15, j = threadIdx.x & 15;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float a0 = t == j ? 1.f : 0.f, a1 = 0.f;
      const float4* row = reinterpret_cast<const float4*>(A + (b + t) * L::AP + b);
#pragma unroll
      for (int q = 0; q < (t + 3) / 4; ++q) {
        const float4 c = row[q];                           // entries at and after the diagonal are zero
        a0 = fmaf(-c.x, x[4 * q], a0);
        if (4 * q + 1 < t) a1 = fmaf(-c.y, x[4 * q + 1], a1);
        if (4 * q + 2 < t) a0 = fmaf(-c.z, x[4 * q + 2], a0);
        if (4 * q + 3 < t) a1 = fmaf(-c.w, x[4 * q + 3], a1);
      }
      x[t] = a0 + a1;
      I[(b + t) * L::AP + b + j] = x[t];
    }
  } else if (threadIdx.x >= 128 && threadIdx.x < 128 + CQ) {
    const int t = threadIdx.x - 128;
    float* v = reinterpret_cast<float*>(ws + 2 * FRAG_BYTES);
    const float e = ex2(vL[t]), last = vL[CQ - 1];
    v[t] = e * rk[t];
    v[CQ + t] = e * rq[t];
    v[2 * CQ + t] = vb[t];
    v[3 * CQ + t] = ex2(last - vL[t]) * rk[t];
    if (t == 0) v[4 * CQ] = ex2(last);
  }
  __syncthreads();
  {
    const int r = threadIdx.x >> 4, c = threadIdx.x & 15;
    auto row_dot = [&](const float* row, const float* col) {       // 16 elements of a row and of a column
      float a0 = 0.f, a1 = 0.f;
#pragma unroll
      for (int m = 0; m < 16; m += 4) {
        const float4 f = *reinterpret_cast<const float4*>(row + m);
        a0 = fmaf(f.x, col[m * L::AP], a0);
        a1 = fmaf(f.y, col[(m + 1) * L::AP], a1);
        a0 = fmaf(f.z, col[(m + 2) * L::AP], a0);
        a1 = fmaf(f.w, col[(m + 3) * L::AP], a1);
      }
      return a0 + a1;
    };
#pragma unroll
    for (int dist = 1; dist < 4; ++dist) {
      float y[3];
#pragma unroll
      for (int bj = 0; bj + dist < 4; ++bj) {
        float sum = 0.f;
#pragma unroll
        for (int k = bj; k < bj + dist; ++k)
          sum += row_dot(A + ((bj + dist) * 16 + r) * L::AP + k * 16, I + k * 16 * L::AP + bj * 16 + c);
        I[((bj + dist) * 16 + r) * L::AP + bj * 16 + c] = sum;
      }
      __syncthreads();
#pragma unroll
      for (int bj = 0; bj + dist < 4; ++bj)
        y[bj] = -row_dot(I + ((bj + dist) * 16 + r) * L::AP + (bj + dist) * 16, I + (bj + dist) * 16 * L::AP + bj * 16 + c);
      __syncthreads();
#pragma unroll
      for (int bj = 0; bj + dist < 4; ++bj) I[((bj + dist) * 16 + r) * L::AP + bj * 16 + c] = y[bj];
      __syncthreads();
    }
  }
  uint4* frag = reinterpret_cast<uint4*>(ws);
  for (int i = warp; i < 16; i += 8) {
    const int w = i >> 2, kb = i & 3;
    if (kb > w) continue;
    const float* a = I + (w * 16 + (lane >> 2)) * L::AP + kb * 16 + (lane & 3) * 2;
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int z = 0; z < 4; ++z) {
      const float2 f = *reinterpret_cast<const float2*>(a + (z & 1) * 8 * L::AP + (z >> 1) * 8);
      split_pair(f.x, f.y, hi[z], lo[z]);
    }
    uint4* o = frag + (i * 32 + lane) * 2;
    o[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    o[1] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
}

// CTA = (32 columns of P, head, sequence). Warps 0-3: outputs of 16 tokens each; warps 4-7: the u of 16 tokens each and the state,
// NT / 4 rows each in their accumulators. Two CTA-wide barriers per chunk: operands are there; the u are there and the old state
// operand has been read.
template <int NT>
struct DeltaSmem {
  static constexpr int NP = NT + 8, QK = CQ * NP * 2, V = CQ * CPP * 2;
  static constexpr int K = 0, Q = 2 * QK, VV = Q + QK, VEC = VV + 2 * V, S = VEC + 2 * VEC_FLOATS * 4, U = S + 2 * NT * CPP * 2, R = U + 2 * V,
                       BYTES = R + 2 * V;
};
template <int NT>
__global__ void __launch_bounds__(256, NT <= 128 ? 2 : 1) delta_chunk_kernel(const DeltaParams p, int slices, int conv_parts) {
  using L = DeltaSmem<NT>;
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
  auto load = [&](int i, int t0) {                         // keys, values and vectors of chunk i
    load_rows<NT>(sb + L::K + (i & 1) * L::QK, k, p.k_ld, t0, n, p.N, threadIdx.x, 256);
    const int r = threadIdx.x / (CP / 8), c = threadIdx.x % (CP / 8);      // 64 rows x 4 pieces
    const bool ok = t0 + r < n && c * 8 < ncol;
    cp_async16(sb + L::VV + (i & 1) * L::V + (r * CPP + c * 8) * 2, ok ? v + (t0 + r) * p.v_ld + c * 8 : v, ok);
    if (threadIdx.x < VEC_FLOATS / 4)
      cp_async16(sb + L::VEC + (i & 1) * (VEC_FLOATS * 4) + threadIdx.x * 16, chunk_ws(p, row0, s, i, h) + 2 * FRAG_BYTES + threadIdx.x * 16, true);
    cp_async_commit();
  };
  auto vec = [&](int i) { return reinterpret_cast<const float*>(smem + L::VEC + (i & 1) * (VEC_FLOATS * 4)); };
  // acc (16 rows from the A-fragments of a block row) += F X, both hi + lo; X [64][CPP] at smem offset x
  auto mul_frags = [&](float (&acc)[CP / 8][4], const uint4 (&f)[4][2], uint32_t x, int w) {
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      if (kb > w) break;
      const uint32_t hi[4] = {f[kb][0].x, f[kb][0].y, f[kb][0].z, f[kb][0].w}, lo[4] = {f[kb][1].x, f[kb][1].y, f[kb][1].z, f[kb][1].w};
      const uint32_t xa = sb + x + ((kb * 16 + (lane & 15)) * CPP + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int j = 0; j < CP / 16; ++j) {
        uint32_t b[4], c[4];
        ldsm4_t(b, xa + j * 32);
        ldsm4_t(c, xa + L::V + j * 32);
        mma_bf16(acc[2 * j], hi, b[0], b[1]);
        mma_bf16(acc[2 * j + 1], hi, b[2], b[3]);
        mma_bf16(acc[2 * j], lo, b[0], b[1]);
        mma_bf16(acc[2 * j + 1], lo, b[2], b[3]);
        mma_bf16(acc[2 * j], hi, c[0], c[1]);
        mma_bf16(acc[2 * j + 1], hi, c[2], c[3]);
      }
    }
  };
  auto load_frags = [&](uint4 (&f)[4][2], const uint8_t* at, int w) {
    const uint4* src = reinterpret_cast<const uint4*>(at) + (w * 4 * 32 + lane) * 2;
#pragma unroll
    for (int kb = 0; kb < 4; ++kb)
      if (kb <= w) {
        f[kb][0] = src[kb * 64];
        f[kb][1] = src[kb * 64 + 1];
      }
  };
  // acc (16 rows of raw keys or queries) = X S with the state operand
  auto mul_state = [&](float (&acc)[CP / 8][4], const uint32_t (&f)[NT / 16][4]) {
    const uint32_t sa = sb + L::S + ((lane & 15) * CPP + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[j][x] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NT / 16; ++kk)
#pragma unroll
      for (int x = 0; x < 2; ++x)                          // hi, lo
#pragma unroll
        for (int j = 0; j < CP / 16; ++j) {
          uint32_t b[4];
          ldsm4_t(b, sa + x * (NT * CPP * 2) + (kk * 16 * CPP + j * 16) * 2);
          mma_bf16(acc[2 * j], f[kk], b[0], b[1]);
          mma_bf16(acc[2 * j + 1], f[kk], b[2], b[3]);
        }
  };
  const int w = warp & 3, tr = w * 16 + (lane >> 2), scol = (lane & 3) * 2;
  load(0, 0);

  if (warp < 4) {
    load_rows<NT>(sb + L::Q, q, p.q_ld, 0, n, p.N, threadIdx.x, 128);
    cp_async_commit();
    int it = 0;
    for (int t0 = 0; t0 < n; t0 += CQ, ++it) {
      cp_async_wait<0>();
      __syncthreads();
      if (t0 + CQ < n) load(it + 1, t0 + CQ);
      uint4 mf[4][2];
      load_frags(mf, chunk_ws(p, row0, s, it, h) + FRAG_BYTES, w);
      uint32_t qf[NT / 16][4];
      const uint32_t qa = sb + L::Q + ((w * 16 + (lane & 15)) * L::NP + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int kk = 0; kk < NT / 16; ++kk) ldsm4(qf[kk], qa + kk * 32);
      asm volatile("bar.sync 3, 128;" ::: "memory");       // every query is in registers
      if (t0 + CQ < n) {
        load_rows<NT>(sb + L::Q, q, p.q_ld, t0 + CQ, n, p.N, threadIdx.x, 128);
        cp_async_commit();
      }
      float o[CP / 8][4];
      mul_state(o, qf);
      const float* vc = vec(it);
      const float gq[2] = {vc[CQ + tr], vc[CQ + tr + 8]};
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) o[j][x] *= gq[x >> 1];
      asm volatile("bar.sync 2, 256;" ::: "memory");
      mul_frags(o, mf, L::U, w);
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int t = tr + 8 * y;
        if (t0 + t >= n) continue;
        bf16* orow = reinterpret_cast<bf16*>(p.out) + (row0 + t0 + t) * p.o_ld + (long long)h * p.P + c0;
#pragma unroll
        for (int j = 0; j < CP / 8; ++j) {
          const int c = j * 8 + scol;
          if (c < ncol) *reinterpret_cast<__nv_bfloat162*>(orow + c) = __floats2bfloat162_rn(o[j][2 * y], o[j][2 * y + 1]);
        }
      }
    }
    return;
  }

  // ---- u and state ----
  constexpr int MT = NT / 64;                              // 16-row state tiles of a warp
  float S[MT][CP / 8][4];
  float* st = p.state + (((long long)(slot < 0 ? 0 : slot) * p.heads + h) * p.N) * p.P + c0;
  const int srow = w * (NT / 4) + (lane >> 2);
  const bool have = slot >= 0 && start > 0;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int r = srow + i * 16 + 8 * y, c = j * 8 + scol;
        const bool ok = have && r < p.N && c < ncol;       // ncol is a multiple of 8
        S[i][j][2 * y] = ok ? st[(long long)r * p.P + c] : 0.f;
        S[i][j][2 * y + 1] = ok ? st[(long long)r * p.P + c + 1] : 0.f;
      }
  auto publish = [&]() {                                   // S as hi / lo operands
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
  auto put_rows = [&](int at, const float (&a)[CP / 8][4], float f0, float f1) {          // rows tr, tr + 8 as hi / lo operands
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        uint32_t hi, lo;
        split_pair(a[j][2 * y] * (y ? f1 : f0), a[j][2 * y + 1] * (y ? f1 : f0), hi, lo);
        const int off = ((tr + 8 * y) * CPP + j * 8 + scol) * 2;
        *reinterpret_cast<uint32_t*>(smem + at + off) = hi;
        *reinterpret_cast<uint32_t*>(smem + at + L::V + off) = lo;
      }
  };
  publish();
  int it = 0;
  for (int t0 = 0; t0 < n; t0 += CQ, ++it) {
    cp_async_wait<0>();
    __syncthreads();
    if (t0 + CQ < n) load(it + 1, t0 + CQ);
    uint4 tf[4][2];
    load_frags(tf, chunk_ws(p, row0, s, it, h), w);
    const uint32_t kbase = sb + L::K + (it & 1) * L::QK;
    const float* vc = vec(it);
    float a[CP / 8][4];
    {
      uint32_t kf[NT / 16][4];
      const uint32_t ka = kbase + ((w * 16 + (lane & 15)) * L::NP + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int kk = 0; kk < NT / 16; ++kk) ldsm4(kf[kk], ka + kk * 32);
      mul_state(a, kf);
    }
    const bf16* sv = reinterpret_cast<const bf16*>(smem + L::VV + (it & 1) * L::V);
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const float gk = vc[tr + 8 * y];
#pragma unroll
      for (int j = 0; j < CP / 8; ++j) {
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + (tr + 8 * y) * CPP + j * 8 + scol));
        a[j][2 * y] = x.x - gk * a[j][2 * y];
        a[j][2 * y + 1] = x.y - gk * a[j][2 * y + 1];
      }
    }
    put_rows(L::R, a, vc[2 * CQ + tr], vc[2 * CQ + tr + 8]);
    asm volatile("bar.sync 1, 128;" ::: "memory");         // right-hand sides written
#pragma unroll
    for (int j = 0; j < CP / 8; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) a[j][x] = 0.f;
    mul_frags(a, tf, L::R, w);
    put_rows(L::U, a, 1.f, 1.f);
    asm volatile("bar.sync 1, 128;" ::: "memory");         // right-hand sides read: their place takes the state's share of u
    put_rows(L::R, a, vc[3 * CQ + tr], vc[3 * CQ + tr + 8]);
    const float keep = vc[4 * CQ];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < CP / 8; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) S[i][j][x] *= keep;
    asm volatile("bar.sync 2, 256;" ::: "memory");
#pragma unroll
    for (int kb = 0; kb < CQ / 16; ++kb) {
      uint32_t b[2][CP / 16][4];
      const uint32_t wa = sb + L::R + ((kb * 16 + (lane & 15)) * CPP + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int j = 0; j < CP / 16; ++j) ldsm4_t(b[x][j], wa + x * L::V + j * 32);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        uint32_t kt[4];                                    // A = K^T: rows n, columns s, read transposed from K [s][n]
        ldsm4_t(kt, kbase + ((kb * 16 + (lane & 7) + ((lane >> 4) << 3)) * L::NP + w * (NT / 4) + i * 16 + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
          for (int j = 0; j < CP / 16; ++j) {
            mma_bf16(S[i][2 * j], kt, b[x][j][0], b[x][j][1]);
            mma_bf16(S[i][2 * j + 1], kt, b[x][j][2], b[x][j][3]);
          }
      }
    }
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
  }
}

template <typename T>
int launch_tokens(const DeltaParams& p, int nseq, cudaStream_t st) {
  const int slices = (p.P + 31) / 32;
  const int conv_parts = p.conv_state ? (p.conv_C + 2047) / 2048 : 0;
  const dim3 grid(slices + conv_parts, p.heads, nseq);
  const long long rows = p.nd > 0 && p.seq0 + nseq <= p.nd ? p.nd : 1 << 20;     // a programmatic dependent launch only pays in decode-sized steps
#define DELTA_CASE(NR)                                                                                           \
  if (p.N <= 8 * NR) {                                                                                           \
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, delta_kernel<T, NR>, grid, dim3(256), 0, st, p, slices, conv_parts));   \
    dlti_count_launch();                                                                                         \
    return 0;                                                                                                    \
  }
  DELTA_CASE(4) DELTA_CASE(8) DELTA_CASE(16) DELTA_CASE(32) DELTA_CASE(64)
#undef DELTA_CASE
  dlti_set_error("delta_scan: keys of up to 512 dimensions");
  return DLTI_ERR_TOO_LARGE;
}

template <int NT>
int launch_chunks(const DeltaParams& p, int nseq, int longest, cudaStream_t st) {
  static bool done[64] = {};
  int dev = 0;
  DLTI_CUDA_CHECK(cudaGetDevice(&dev));
  if (!done[dev & 63]) {
    DLTI_CUDA_CHECK(cudaFuncSetAttribute(delta_prep_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, PrepSmem<NT>::BYTES));
    DLTI_CUDA_CHECK(cudaFuncSetAttribute(delta_chunk_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, DeltaSmem<NT>::BYTES));
    done[dev & 63] = true;
  }
  const int slices = (p.P + CP - 1) / CP;
  const int conv_parts = p.conv_state ? (p.conv_C + 2047) / 2048 : 0;
  delta_prep_kernel<NT><<<dim3((longest + CQ - 1) / CQ, p.heads, nseq), 256, PrepSmem<NT>::BYTES, st>>>(p);
  DLTI_CUDA_CHECK(cudaGetLastError());
  delta_chunk_kernel<NT><<<dim3(slices + conv_parts, p.heads, nseq), 256, DeltaSmem<NT>::BYTES, st>>>(p, slices, conv_parts);
  dlti_count_launch(2);
  return (int)cudaGetLastError();
}

}  // namespace

// bytes that the chunked form needs for `rows` prompt rows of nseq sequences
DLTI_API long long dlti_delta_workspace(long long rows, int nseq, int heads) {
  return (chunk_base(rows, nseq) + 1) * (long long)heads * WS_BYTES;
}

// Sequences [seq0, seq0 + nseq) of the step. ws null: token by token (N <= 512); else the chunked form for prompt sequences of at
// most `longest` rows (seq0 = nd; bf16, N and P multiples of 8, N <= 256, 16-byte aligned rows). conv_*: see conv_tail.
DLTI_API int dlti_delta_scan(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, const float* gates,
                             long long g_ld, const float* A_log, const float* dt_bias, float* state, const int* sslot, const int* ctx,
                             const int* cu, int nd, int seq0, int nseq, int heads, int groups, int N, int P, void* out, long long o_ld,
                             const void* conv_src, long long conv_ld, int conv_col, int conv_rows, int conv_C, void* conv_state, void* ws,
                             int longest, int dtype, cudaStream_t st) {
  if (nseq <= 0) return 0;
  if (heads < 1 || groups < 1 || heads % groups || N < 1 || P < 1 || nseq > 65535 || !gates || !A_log || !dt_bias) return DLTI_ERR_BAD_ARG;
  if (conv_rows <= 0) conv_state = nullptr;
  DeltaParams p{q, k, v, q_ld, k_ld, v_ld, gates, g_ld, A_log, dt_bias, state, sslot, ctx, cu, nd, seq0, heads, heads / groups, N, P, out, o_ld,
                conv_src, conv_ld, conv_col, conv_rows, conv_C, conv_state, (uint8_t*)ws};
  if (!ws) {
    if (dtype == DLTI_BF16) return launch_tokens<__nv_bfloat16>(p, nseq, st);
    if (dtype == DLTI_FP32) return launch_tokens<float>(p, nseq, st);
    return DLTI_ERR_UNSUPPORTED;
  }
  if (dtype != DLTI_BF16 || seq0 < nd || longest < 1 || N % 8 || P % 8 || q_ld % 8 || k_ld % 8 || v_ld % 8 || o_ld % 2 ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(ws)) & 15)) {
    dlti_set_error("delta_scan, chunked: bf16, 16-byte aligned rows, N and P multiples of 8");
    return DLTI_ERR_BAD_ARG;
  }
  if (N <= 64) return launch_chunks<64>(p, nseq, longest, st);
  if (N <= 128) return launch_chunks<128>(p, nseq, longest, st);
  if (N <= 256) return launch_chunks<256>(p, nseq, longest, st);
  dlti_set_error("delta_scan, chunked: keys of up to 256 dimensions");
  return DLTI_ERR_TOO_LARGE;
}

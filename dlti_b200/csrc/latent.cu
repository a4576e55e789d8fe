// Latent attention: every token caches one row [c | k_rot], the normed latent c (rank numbers) and a rotated key part that
// all heads share; a head's keys and values are linear in c (K_h = Uk_h c, V_h = Uv_h c).
//
//   latent_prep      projection row -> rotated queries, cache row (latent norm, rotated key part), head gates
//   head_gemm        per-head matrix products: queries into the latent space (q Uk_h), latent outputs to values (Uv_h o)
//   latent_decode    absorbed form: scores of all heads against the cached rows themselves, values = their first rank
//                    columns; each cached row is read once for all heads of a block
//
// Prompts take the expanded form instead: keys and values of all heads by one GEMM from the cached rows (an identity block
// in its weight passes k_rot through), then ordinary causal attention (attention.cu, attention_paged.cu).
//
// A cache row is [c, zeros to a multiple of 16, k_rot, zeros to a multiple of 16, 8 zeros]: rot_at = round16(rank) and
// pitch = rot_at + round16(rot) + 8. The last 8 make the rows of a page lie in shared memory, copied in one piece, so that
// ldmatrix reads eight of them without bank conflicts.
#include "rows.cuh"
#include "mma_sync.cuh"

namespace {

using bf16 = __nv_bfloat16;
constexpr float LOG2E_F = 1.4426950408889634f;

struct PrepParams {
  const void* proj; long long ld; int oq, od, og;          // section columns: queries, latent | shared key part, gates (< 0: none)
  int H, dim, rot, rank, rd, interleaved;                  // rd: rotated dimensions of rot
  const float *cos_t, *sin_t; const int* pos;
  const float* kvw; float eps;
  const long long* slots; void* cache; int pitch, rot_at;
  int nabs;                                                // rows below: absorbed form; from there on: expanded form
  void* qn; int qn_hd;                                     // absorbed: unrotated queries [nabs, H, qn_hd]
  void* ql;                                                // absorbed: [nabs, H, pitch], here the rotated part and the padding
  void* qp; long long qp_ld; int qp_hd;                    // expanded: [dim | rot | zeros] per head, row qdst[t - nabs]
  void* lat;                                               // expanded: the cache rows again [., pitch], row dst[t - nabs]
  const int *qdst, *dst;                                   // null: t - nabs
  float* gate;
  long long tokens;
};

template <typename T>
__device__ __forceinline__ void zero8(T* p) {
  const float z[8] = {};
  put_n<T, 8>(p, z);
}

// sizes, sections and pitches multiples of 8, interleaved pairs, rank <= 1024. Block y = 0: warp 0 the cache row, warp 1 the
// gates; the others 128 * QP pieces of 8 query columns.
template <bool ACC, int QP>
__global__ void __launch_bounds__(128) latent_prep_vec_kernel(const PrepParams p, int units, int per_head) {
  using T = bf16;
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  const uint8_t* row = reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * (ACC ? 4 : sizeof(T));
  const int ps = p.pos[t], half = p.rd >> 1, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool expanded = t >= p.nabs;
  const long long to = expanded ? (p.dst ? (long long)p.dst[t - p.nabs] : t - p.nabs) : 0;
  const long long tq = expanded ? (p.qdst ? (long long)p.qdst[t - p.nabs] : t - p.nabs) : 0;
  auto rotate8 = [&](float (&f)[8], int e0) {              // e0: offset in the rotated part
    if (e0 >= p.rd) return;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float c = p.cos_t[(long long)ps * half + e0 / 2 + j], s = p.sin_t[(long long)ps * half + e0 / 2 + j];
      const float a = f[2 * j], b = f[2 * j + 1];
      f[2 * j] = a * c - b * s;
      f[2 * j + 1] = b * c + a * s;
    }
  };
  if (blockIdx.y == 0) {
    if (warp == 0) {
      const long long slot = p.slots[t];
      T* dst0 = slot >= 0 ? reinterpret_cast<T*>(p.cache) + slot * p.pitch : nullptr;
      T* dst1 = expanded ? reinterpret_cast<T*>(p.lat) + to * p.pitch : nullptr;
      float f[4][8];
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int e = (lane + 32 * i) * 8;
        if (e < p.rank) {
          take_n<T, ACC, 8>(row, p.od + e, f[i]);
#pragma unroll
          for (int j = 0; j < 8; ++j) ss += f[i][j] * f[i][j];
        }
      }
      const float r = 1.f / sqrtf(warp_sum(ss) / (float)p.rank + p.eps);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int e = (lane + 32 * i) * 8;
        if (e < p.rank) {
          float w[8];
          ld8(p.kvw + e, w);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[i][j] *= r * w[j];
          if (dst0) put_n<T, 8>(dst0 + e, f[i]);
          if (dst1) put_n<T, 8>(dst1 + e, f[i]);
        }
      }
      for (int e = lane * 8; e < p.pitch - p.rank; e += 256) {       // [rank, rot_at): zeros, then k_rot, then zeros
        const int c = p.rank + e, k = c - p.rot_at;
        float g[8] = {};
        if (k >= 0 && k < p.rot) {
          take_n<T, ACC, 8>(row, p.od + p.rank + k, g);
          rotate8(g, k);
        }
        if (dst0) put_n<T, 8>(dst0 + c, g);
        if (dst1) put_n<T, 8>(dst1 + c, g);
      }
    } else if (warp == 1 && p.og >= 0) {
      for (int h = lane; h < p.H; h += 32) p.gate[t * p.H + h] = sigmoid_f(take<T, ACC>(row, p.og + h));
    }
    return;
  }
  const int ph = (p.dim + p.rot) >> 3;
  float f[QP][8];
  int head[QP], u[QP];
#pragma unroll
  for (int i = 0; i < QP; ++i) {
    const int x = (blockIdx.y - 1) * 128 * QP + i * 128 + threadIdx.x;
    head[i] = x < units ? x / per_head : -1;
    u[i] = x - head[i] * per_head;
    if (head[i] >= 0 && u[i] < ph) take_n<T, ACC, 8>(row, p.oq + (head[i] * ph + u[i]) * 8, f[i]);
  }
#pragma unroll
  for (int i = 0; i < QP; ++i) {
    if (head[i] < 0) continue;
    const int e = u[i] * 8;
    if (u[i] < ph) {
      if (e >= p.dim) rotate8(f[i], e - p.dim);
      T* o;
      if (expanded) o = reinterpret_cast<T*>(p.qp) + tq * p.qp_ld + (long long)head[i] * p.qp_hd + e;
      else if (e < p.dim) o = reinterpret_cast<T*>(p.qn) + (t * p.H + head[i]) * p.qn_hd + e;
      else o = reinterpret_cast<T*>(p.ql) + (t * p.H + head[i]) * p.pitch + p.rot_at + e - p.dim;
      put_n<T, 8>(o, f[i]);
    } else if (expanded) {
      if (e < p.qp_hd) zero8(reinterpret_cast<T*>(p.qp) + tq * p.qp_ld + (long long)head[i] * p.qp_hd + e);
    } else {
      int c = p.rank + (u[i] - ph) * 8;                    // [rank, rot_at), then [rot_at + rot, pitch)
      if (c >= p.rot_at) c += p.rot;
      if (c < p.pitch) zero8(reinterpret_cast<T*>(p.ql) + (t * p.H + head[i]) * p.pitch + c);
    }
  }
}

// any sizes: one CTA per token
template <typename T, bool ACC>
__global__ void __launch_bounds__(128) latent_prep_kernel(const PrepParams p) {
  __shared__ float red[32];
  extern __shared__ float cs[];                            // [rank]
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  const uint8_t* row = reinterpret_cast<const uint8_t*>(p.proj) + t * p.ld * (ACC ? 4 : sizeof(T));
  const int ps = p.pos[t], half = p.rd >> 1, npair = half + ((p.rot - p.rd + 1) >> 1), qh = p.dim + p.rot;
  const bool expanded = t >= p.nabs;
  const long long to = expanded ? (p.dst ? (long long)p.dst[t - p.nabs] : t - p.nabs) : 0;
  const long long tq = expanded ? (p.qdst ? (long long)p.qdst[t - p.nabs] : t - p.nabs) : 0;
  // pair j of a rotated part that starts at column col of the row -> o[...]
  auto pair = [&](int col, int j, T* o, T* o2) {
    const int e0 = j < half ? (p.interleaved ? 2 * j : j) : p.rd + 2 * (j - half);
    const int e1 = j < half ? (p.interleaved ? 2 * j + 1 : j + half) : e0 + 1;
    float a = take<T, ACC>(row, col + e0), b = e1 < p.rot ? take<T, ACC>(row, col + e1) : 0.f;
    if (j < half) {
      const float c = p.cos_t[(long long)ps * half + j], s = p.sin_t[(long long)ps * half + j];
      const float u = a * c - b * s;
      b = b * c + a * s;
      a = u;
    }
    if (o) { o[e0] = Cvt<T>::from_f(a); if (e1 < p.rot) o[e1] = Cvt<T>::from_f(b); }
    if (o2) { o2[e0] = Cvt<T>::from_f(a); if (e1 < p.rot) o2[e1] = Cvt<T>::from_f(b); }
  };
  T* qp = expanded ? reinterpret_cast<T*>(p.qp) + tq * p.qp_ld : nullptr;
  T* qn = expanded ? nullptr : reinterpret_cast<T*>(p.qn) + t * p.H * p.qn_hd;
  T* ql = expanded ? nullptr : reinterpret_cast<T*>(p.ql) + t * p.H * p.pitch;
  for (int i = threadIdx.x; i < p.H * p.dim; i += blockDim.x) {
    const int h = i / p.dim, e = i - h * p.dim;
    const T v = Cvt<T>::from_f(take<T, ACC>(row, p.oq + h * qh + e));
    if (expanded) qp[(long long)h * p.qp_hd + e] = v;
    else qn[h * p.qn_hd + e] = v;
  }
  for (int i = threadIdx.x; i < p.H * npair; i += blockDim.x) {
    const int h = i / npair;
    pair(p.oq + h * qh + p.dim, i - h * npair, expanded ? qp + (long long)h * p.qp_hd + p.dim : ql + (long long)h * p.pitch + p.rot_at, nullptr);
  }
  const T z = Cvt<T>::from_f(0.f);
  if (expanded) {
    const int pad = p.qp_hd - qh;
    for (int i = threadIdx.x; i < p.H * pad; i += blockDim.x) qp[(long long)(i / pad) * p.qp_hd + qh + i % pad] = z;
  } else {
    const int pad = p.pitch - p.rank - p.rot;
    for (int i = threadIdx.x; i < p.H * pad; i += blockDim.x) {
      int c = p.rank + i % pad;
      if (c >= p.rot_at) c += p.rot;
      ql[(long long)(i / pad) * p.pitch + c] = z;
    }
    for (int i = threadIdx.x; i < p.H * (p.qn_hd - p.dim); i += blockDim.x)
      qn[i / (p.qn_hd - p.dim) * p.qn_hd + p.dim + i % (p.qn_hd - p.dim)] = z;
  }
  if (p.og >= 0)
    for (int h = threadIdx.x; h < p.H; h += blockDim.x) p.gate[t * p.H + h] = sigmoid_f(take<T, ACC>(row, p.og + h));
  const long long slot = p.slots[t];
  T* dst0 = slot >= 0 ? reinterpret_cast<T*>(p.cache) + slot * p.pitch : nullptr;
  T* dst1 = expanded ? reinterpret_cast<T*>(p.lat) + to * p.pitch : nullptr;
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.rank; c += blockDim.x) {
    const float v = cs[c] = take<T, ACC>(row, p.od + c);
    ss += v * v;
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)p.rank + p.eps);
  for (int c = threadIdx.x; c < p.rank; c += blockDim.x) {
    const T v = Cvt<T>::from_f(cs[c] * r * p.kvw[c]);
    if (dst0) dst0[c] = v;
    if (dst1) dst1[c] = v;
  }
  for (int j = threadIdx.x; j < npair; j += blockDim.x) pair(p.od + p.rank, j, dst0 ? dst0 + p.rot_at : nullptr, dst1 ? dst1 + p.rot_at : nullptr);
  for (int i = threadIdx.x; i < p.pitch - p.rank - p.rot; i += blockDim.x) {
    int c = p.rank + i;
    if (c >= p.rot_at) c += p.rot;
    if (dst0) dst0[c] = z;
    if (dst1) dst1[c] = z;
  }
}

// cached rows in front of a portion's own ones: lat[rows[i]] = cache[slots[i]], 16-byte pieces
__global__ void latent_rows_kernel(bf16* __restrict__ lat, const bf16* __restrict__ cache, int pitch, const int* __restrict__ rows,
                                   const int* __restrict__ slots, long long total) {
  const int pieces = pitch / 8;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / pieces;
    const int c = (int)(i - r * pieces) * 8;
    *reinterpret_cast<int4*>(lat + (long long)rows[r] * pitch + c) = *reinterpret_cast<const int4*>(cache + (long long)slots[r] * pitch + c);
  }
}

// out[t, h, n] = sum_k a[t, h, k] B_h(k, n), heads a_hd / o_hd columns apart; B_h is head h's block of K (KN) or N rows of b:
//   KN:  b [H * K, N]   B_h(k, n) = b[h K + k, n]          NK:  b [H * N, K]   B_h(k, n) = b[h N + n, k]
struct HeadGemmParams {
  const void* a; long long a_ld; int a_hd;
  const void* b; long long b_ld;
  void* out; long long o_ld; int o_hd;
  long long rows; int H, K, N;
};
constexpr int HG_M = 64, HG_N = 64, HG_K = 64, HG_P = HG_K + 8, HG_STAGES = 3, HG_STAGE = 2 * 64 * HG_P * 2;
template <bool KN>
__global__ void __launch_bounds__(128) head_gemm_kernel(const HeadGemmParams p) {
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  const int h = blockIdx.y, n0 = blockIdx.x * HG_N, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long t0 = (long long)blockIdx.z * HG_M;
  const bf16* A = reinterpret_cast<const bf16*>(p.a) + t0 * p.a_ld + (long long)h * p.a_hd;
  const bf16* B = reinterpret_cast<const bf16*>(p.b) + (long long)h * (KN ? p.K : p.N) * p.b_ld;
  const int nk = (p.K + HG_K - 1) / HG_K;
  const int lr = threadIdx.x >> 3, lc = (threadIdx.x & 7) * 8;       // 16 rows a pass, 8 pieces a row
  auto load_b = [&](int it) {
    const uint32_t dst = sb + (it % HG_STAGES) * HG_STAGE + 64 * HG_P * 2;
    const int k0 = it * HG_K;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = lr + 16 * i;
      const bool ok = KN ? (k0 + r < p.K && n0 + lc < p.N) : (n0 + r < p.N && k0 + lc < p.K);
      const bf16* src = KN ? B + (long long)(k0 + r) * p.b_ld + n0 + lc : B + (long long)(n0 + r) * p.b_ld + k0 + lc;
      cp_async16(dst + (r * HG_P + lc) * 2, ok ? src : B, ok);
    }
  };
  auto load_a = [&](int it) {
    const uint32_t dst = sb + (it % HG_STAGES) * HG_STAGE;
    const int k0 = it * HG_K;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = lr + 16 * i;
      const bool ok = t0 + r < p.rows && k0 + lc < p.K;
      cp_async16(dst + (r * HG_P + lc) * 2, ok ? A + (long long)r * p.a_ld + k0 + lc : A, ok);
    }
  };
#pragma unroll
  for (int i = 0; i < HG_STAGES - 1; ++i)                  // weights never change: they may come before the wait
    if (i < nk) load_b(i);
  griddep_wait();
  griddep_launch();
#pragma unroll
  for (int i = 0; i < HG_STAGES - 1; ++i) {
    if (i < nk) load_a(i);
    cp_async_commit();
  }
  float o[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int x = 0; x < 4; ++x) o[j][x] = 0.f;
  const bool on = t0 + warp * 16 < p.rows;
  for (int it = 0; it < nk; ++it) {
    cp_async_wait<HG_STAGES - 2>();
    __syncthreads();
    if (it + HG_STAGES - 1 < nk) { load_a(it + HG_STAGES - 1); load_b(it + HG_STAGES - 1); }
    cp_async_commit();
    if (!on) continue;
    const uint32_t sa = sb + (it % HG_STAGES) * HG_STAGE, sB = sa + 64 * HG_P * 2;
#pragma unroll
    for (int kk = 0; kk < HG_K / 16; ++kk) {
      uint32_t a[4];
      ldsm4(a, sa + ((warp * 16 + (lane & 15)) * HG_P + kk * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
      for (int j = 0; j < HG_N / 16; ++j) {
        uint32_t b[4];
        if constexpr (KN) ldsm4_t(b, sB + ((kk * 16 + (lane & 15)) * HG_P + j * 16 + (lane >> 4) * 8) * 2);
        else ldsm4(b, sB + ((j * 16 + (lane & 7) + ((lane >> 4) << 3)) * HG_P + kk * 16 + ((lane >> 3) & 1) * 8) * 2);
        mma_bf16(o[2 * j], a, b[0], b[1]);
        mma_bf16(o[2 * j + 1], a, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    const long long t = t0 + warp * 16 + (lane >> 2) + 8 * y;
    if (t >= p.rows) continue;
    bf16* orow = reinterpret_cast<bf16*>(p.out) + t * p.o_ld + (long long)h * p.o_hd;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int n = n0 + j * 8 + (lane & 3) * 2;           // N is a multiple of 8
      if (n < p.N) *reinterpret_cast<__nv_bfloat162*>(orow + n) = __floats2bfloat162_rn(o[j][2 * y], o[j][2 * y + 1]);
    }
  }
}
// fp32 arithmetic, any sizes: a thread per output
template <typename T, bool KN>
__global__ void __launch_bounds__(128) head_gemm_any_kernel(const HeadGemmParams p) {
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.y, n = blockIdx.x * 128 + threadIdx.x;
  const long long t = blockIdx.z;
  if (n >= p.N) return;
  const T* a = reinterpret_cast<const T*>(p.a) + t * p.a_ld + (long long)h * p.a_hd;
  const T* b = reinterpret_cast<const T*>(p.b) + (KN ? (long long)h * p.K * p.b_ld + n : ((long long)h * p.N + n) * p.b_ld);
  const long long step = KN ? p.b_ld : 1;
  float acc = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += 16) {                   // short partial sums keep the rounding error small
    float s = 0.f;
    for (int k = k0; k < min(p.K, k0 + 16); ++k) s = fmaf(Cvt<T>::to_f(a[k]), Cvt<T>::to_f(b[k * step]), s);
    acc += s;
  }
  reinterpret_cast<T*>(p.out)[t * p.o_ld + (long long)h * p.o_hd + n] = Cvt<T>::from_f(acc);
}

// Absorbed attention, bf16. grid (splits, blocks of 16 HT heads, rows); row b belongs to sequence rseq[b] (null: b) and sees its
// first min(pos[b] + 1, ctx) cached rows (pos null: all ctx). Tiles of 32 cached rows go through three groups of warps that
// work on different tiles at the same time:
//   warp 16       copies the tile's rows from the pages, one bulk copy per page, `stages` tiles ahead
//   warps 0-7     scores (a warp: 16 keys x 16 heads over one of 4 / HT parts of the row's columns), then the softmax weights
//                 as hi + lo bf16 terms, two buffers
//   warps 8-15    outputs: a warp owns W16 groups of 16 latent columns of all heads
// Every wait is bounded: when one runs out the CTA gives up, and its outputs are NaN.
struct LatentParams {
  const void* q;                                           // [rows, H, pitch]
  const void* cache; int pitch, rank;
  const int* tables; int max_blocks, bs;
  const int *ctx, *rseq, *pos;
  int H; float scale;
  const float *sink, *gate;                                // [H] or null, [rows, H] or null
  void* out;                                               // [rows, H, rot_at]
  int o_hd;
};
constexpr int LKT = 32, LSP = LKT + 4, LPP = LKT + 8;      // keys a tile, score and weight row pitches
constexpr int LTHREADS = 17 * 32, LSTAGES = 6;             // most stages
constexpr long long LWAIT = 4000000000LL;                  // ~2 s
template <int HT>
struct LatentSmem {
  static constexpr int ROWS = 16 * HT, SIDES = 4 / HT;
  static constexpr int BARS = 0, ERR = BARS + (2 * LSTAGES + 4) * 8, S = ERR + 16;                // scores [2][SIDES][ROWS][LSP]
  static constexpr int P = S + 2 * SIDES * ROWS * LSP * 4, A = P + 2 * 2 * ROWS * LPP * 2;        // weights [2][hi, lo][ROWS][LPP]
  static constexpr int Q = A + 4 * ROWS * 4;                                                      // factors [2][ROWS], m, l
  static __host__ __device__ int row(int pitch) { return pitch * 2; }
  static __host__ __device__ int bytes(int pitch, int stages) { return Q + (ROWS + stages * LKT) * row(pitch); }
};
template <int HT, int W16>
__global__ void __launch_bounds__(LTHREADS) latent_decode_kernel(const LatentParams p, int splits, int stages, float* __restrict__ part_o,
                                                                float* __restrict__ part_ml) {
  using L = LatentSmem<HT>;
  constexpr int ROWS = L::ROWS, SIDES = L::SIDES, TPR = 256 / ROWS, KPT = LKT / TPR;       // softmax: threads a row, keys a thread
  extern __shared__ __align__(128) uint8_t smem[];
  float* sS = reinterpret_cast<float*>(smem + L::S);
  float* sA = reinterpret_cast<float*>(smem + L::A);
  volatile int* err = reinterpret_cast<volatile int*>(smem + L::ERR);
  const uint32_t sb = smem_u32(smem), sQ = sb + L::Q, sP = sb + L::P;
  const int kp = L::row(p.pitch), stage = LKT * kp;        // bytes
  const uint32_t sK = sQ + ROWS * kp;
  const uint32_t full = sb + L::BARS, empty = full + 8 * LSTAGES, p_full = empty + 8 * LSTAGES, p_free = p_full + 16;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < stages; ++i) {
      mbar_init(full + 8 * i, 1);
      mbar_init(empty + 8 * i, 8);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(p_full + 8 * i, 8);
      mbar_init(p_free + 8 * i, 8);
    }
    *err = 0;
    mbar_fence_init();
  }
  griddep_wait();
  griddep_launch();
  auto wait = [&](uint32_t bar, uint32_t parity) {
    if (!mbar_try_wait(bar, parity)) {
      const long long t0 = clock64();
      while (!mbar_try_wait(bar, parity) && !*err)
        if (clock64() - t0 > LWAIT) *err = 1;
    }
    __syncwarp();
  };
  const int split = blockIdx.x, h0 = blockIdx.y * ROWS, nh = min(ROWS, p.H - h0);
  const long long b = blockIdx.z;
  const int seq = p.rseq ? p.rseq[b] : (int)b;
  const int n = p.pos ? min(p.pos[b] + 1, p.ctx[seq]) : p.ctx[seq];
  const int tiles = (n + LKT - 1) / LKT, per = (tiles + splits - 1) / splits;
  const int jbeg = split * per * LKT, jend = min(n, jbeg + per * LKT);
  const int nt = jbeg < jend ? (jend - jbeg + LKT - 1) / LKT : 0;
  const int n16 = (p.rank + 15) >> 4;
  const int pieces = p.pitch >> 3;
  if (nt > 0 && warp < 16) {
    const bf16* q = reinterpret_cast<const bf16*>(p.q) + (b * p.H + h0) * p.pitch;
    for (int r = warp; r < ROWS; r += 16)
      for (int c = lane; c < pieces; c += 32) cp_async16(sQ + r * kp + c * 16, r < nh ? q + (long long)r * p.pitch + c * 8 : q, r < nh);
    cp_async_commit();
    cp_async_wait<0>();
  }
  __syncthreads();
  float o[HT][W16][8];
#pragma unroll
  for (int t = 0; t < HT; ++t)
#pragma unroll
    for (int i = 0; i < W16; ++i)
#pragma unroll
      for (int x = 0; x < 8; ++x) o[t][i][x] = 0.f;

  if (warp == 16) {
    // ---- copies: the lane of the first row of a page takes all its rows in the tile; rows past the end become zeros ----
    const int* tab = p.tables + (long long)seq * p.max_blocks;
    const int shift = (p.bs & (p.bs - 1)) ? -1 : 31 - __clz(p.bs);
    auto block_of = [&](int j) { return shift < 0 ? j / p.bs : j >> shift; };
    auto entry = [&](int it) { return tab[block_of(min(jbeg + it * LKT + lane, n - 1))]; };
    int page = nt > 0 ? entry(0) : 0;
    for (int it = 0; it < nt; ++it) {
      const int s = it % stages, j = jbeg + it * LKT + lane, rows = min(LKT, jend - (j - lane)), off = j - block_of(j) * p.bs;
      const int next = entry(it + 1);                      // asked for one tile ahead
      if (it >= stages) wait(empty + 8 * s, (it / stages - 1) & 1);
      for (int i = lane; i < (LKT - rows) * pieces; i += 32)
        *reinterpret_cast<uint4*>(smem + (sK - sb) + s * stage + rows * kp + i * 16) = make_uint4(0, 0, 0, 0);
      __syncwarp();
      if (lane == 0) mbar_expect_tx(full + 8 * s, rows * kp);
      __syncwarp();
      if (lane < rows && (lane == 0 || off == 0))
        bulk_load_1d(sK + s * stage + lane * kp, reinterpret_cast<const bf16*>(p.cache) + ((long long)page * p.bs + off) * p.pitch,
                     min(p.bs - off, rows - lane) * kp, full + 8 * s);
      page = next;
    }
  } else if (warp < 8) {
    // ---- scores and weights ----
    const int ksteps = (p.pitch - 8) >> 4, kpart = (ksteps + SIDES - 1) / SIDES;
    const int kb = (warp & 1) * 16, ht = (warp >> 1) % HT, kside = (warp >> 1) / HT;
    const int k0 = kside * kpart, k1 = min(ksteps, k0 + kpart);
    const int row = threadIdx.x / TPR, key0 = (threadIdx.x % TPR) * KPT;
    const uint32_t qa = sQ + (ht * 16 + (lane & 15)) * kp + (lane >> 4) * 16;
    const uint32_t ka = (kb + (lane & 7) + ((lane >> 4) << 3)) * kp + ((lane >> 3) & 1) * 16;
    const float sl2 = p.scale * LOG2E_F;
    float m = -INFINITY, l = 0.f;
    for (int it = 0; it < nt; ++it) {
      const int s = it % stages, j0 = jbeg + it * LKT, u = it & 1;
      wait(full + 8 * s, (it / stages) & 1);
      const uint32_t kt = sK + s * stage + ka;
      float c[2][2][4] = {};                               // even and odd steps: two chains
#pragma unroll 2
      for (int kk = k0; kk + 1 < k1; kk += 2)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          uint32_t a[4], bb[4];
          ldsm4(bb, kt + (kk + y) * 32);
          ldsm4(a, qa + (kk + y) * 32);
          mma_bf16(c[y][0], a, bb[0], bb[1]);
          mma_bf16(c[y][1], a, bb[2], bb[3]);
        }
      if ((k1 - k0) & 1 && k1 > k0) {
        uint32_t a[4], bb[4];
        ldsm4(bb, kt + (k1 - 1) * 32);
        ldsm4(a, qa + (k1 - 1) * 32);
        mma_bf16(c[0][0], a, bb[0], bb[1]);
        mma_bf16(c[0][1], a, bb[2], bb[3]);
      }
      float* sp = sS + ((u * SIDES + kside) * ROWS + ht * 16 + (lane >> 2)) * LSP + kb + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int y = 0; y < 2; ++y)
          *reinterpret_cast<float2*>(sp + 8 * y * LSP + i * 8) = make_float2(c[0][i][2 * y] + c[1][i][2 * y], c[0][i][2 * y + 1] + c[1][i][2 * y + 1]);
      asm volatile("bar.sync 1, 256;" ::: "memory");       // scores of this tile are written; those of the last one have been read
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        float x = 0.f;
#pragma unroll
        for (int y = 0; y < SIDES; ++y) x += sS[((u * SIDES + y) * ROWS + row) * LSP + key0 + i];
        v[i] = j0 + key0 + i < jend ? x * sl2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int d = TPR / 2; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float nm = fmaxf(m, mx);                       // finite: the tile has a visible key
      const float alpha = ex2(m - nm);
      m = nm;
      l *= alpha;
      if (it >= 2) wait(p_free + 8 * u, ((it >> 1) - 1) & 1);
      if (threadIdx.x % TPR == 0) sA[u * ROWS + row] = alpha;
      bf16* pr = reinterpret_cast<bf16*>(smem + L::P) + (u * 2 * ROWS + row) * LPP + key0;
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const float e0 = ex2(v[i] - nm), e1 = ex2(v[i + 1] - nm);
        l += e0 + e1;
        uint32_t hi, lo;
        split_pair(e0, e1, hi, lo);
        *reinterpret_cast<uint32_t*>(pr + i) = hi;
        *reinterpret_cast<uint32_t*>(pr + ROWS * LPP + i) = lo;
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full + 8 * u);
    }
#pragma unroll
    for (int d = TPR / 2; d > 0; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
    if (threadIdx.x % TPR == 0) {
      sA[2 * ROWS + row] = m;
      sA[3 * ROWS + row] = l;
    }
  } else {
    // ---- outputs ----
    for (int it = 0; it < nt; ++it) {
      const int s = it % stages, u = it & 1;
      wait(full + 8 * s, (it / stages) & 1);
      wait(p_full + 8 * u, (it >> 1) & 1);
      const uint32_t vt = sK + s * stage + (lane & 15) * kp + (lane >> 4) * 16;
#pragma unroll
      for (int t = 0; t < HT; ++t) {
        const float a0 = sA[u * ROWS + t * 16 + (lane >> 2)], a1 = sA[u * ROWS + t * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int i = 0; i < W16; ++i)
#pragma unroll
          for (int x = 0; x < 8; ++x) o[t][i][x] *= (x & 2) ? a1 : a0;
      }
#pragma unroll
      for (int ks = 0; ks < LKT / 16; ++ks) {
        uint32_t w[HT][2][4];
#pragma unroll
        for (int t = 0; t < HT; ++t)
#pragma unroll
          for (int x = 0; x < 2; ++x)
            ldsm4(w[t][x], sP + (((u * 2 + x) * ROWS + t * 16 + (lane & 15)) * LPP + ks * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
        for (int i = 0; i < W16; ++i) {
          const int c16 = (warp - 8) * W16 + i;
          if (c16 >= n16) break;                           // warp-uniform
          uint32_t bb[4];
          ldsm4_t(bb, vt + ks * 16 * kp + c16 * 32);
#pragma unroll
          for (int t = 0; t < HT; ++t)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
              mma_bf16(*reinterpret_cast<float(*)[4]>(&o[t][i][0]), w[t][x], bb[0], bb[1]);
              mma_bf16(*reinterpret_cast<float(*)[4]>(&o[t][i][4]), w[t][x], bb[2], bb[3]);
            }
        }
      }
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(p_free + 8 * u);
        mbar_arrive(empty + 8 * s);
      }
    }
  }
  __syncthreads();                                         // m and l are written
  if (warp < 8 || warp == 16) return;
  const float bad = *err ? __int_as_float(0x7fc00000) : 0.f;
#pragma unroll
  for (int t = 0; t < HT; ++t)
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int r = t * 16 + (lane >> 2) + 8 * y, h = h0 + r;
      if (r >= nh) continue;
      const float mr = sA[2 * ROWS + r], lr = sA[3 * ROWS + r] + bad;
      if (splits == 1) {
        const float d = p.sink ? lr + ex2(p.sink[h] * LOG2E_F - (mr == -INFINITY ? 0.f : mr)) : lr;
        float f = d == 0.f ? 0.f : 1.f / d;
        if (p.gate) f *= p.gate[b * p.H + h];
        bf16* orow = reinterpret_cast<bf16*>(p.out) + (b * p.H + h) * p.o_hd;
#pragma unroll
        for (int i = 0; i < W16; ++i) {
          const int c = ((warp - 8) * W16 + i) * 16 + (lane & 3) * 2;
          if ((warp - 8) * W16 + i >= n16) break;
#pragma unroll
          for (int x = 0; x < 2; ++x)
            *reinterpret_cast<__nv_bfloat162*>(orow + c + 8 * x) = __floats2bfloat162_rn(o[t][i][4 * x + 2 * y] * f, o[t][i][4 * x + 2 * y + 1] * f);
        }
      } else {
        const long long idx = (b * p.H + h) * splits + split;
        if (warp == 8 && (lane & 3) == 0) {
          part_ml[idx * 2] = mr;
          part_ml[idx * 2 + 1] = lr;
        }
#pragma unroll
        for (int i = 0; i < W16; ++i) {
          const int c = ((warp - 8) * W16 + i) * 16 + (lane & 3) * 2;
          if ((warp - 8) * W16 + i >= n16) break;
#pragma unroll
          for (int x = 0; x < 2; ++x)
            *reinterpret_cast<float2*>(part_o + idx * p.o_hd + c + 8 * x) = make_float2(o[t][i][4 * x + 2 * y], o[t][i][4 * x + 2 * y + 1]);
        }
      }
    }
}

// sum of the splits of every (row, head): four latent columns a thread
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentParams p, int splits, const float* __restrict__ part_o,
                                                            const float* __restrict__ part_ml) {
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.x;
  const long long b = blockIdx.y, base = (b * p.H + h) * splits;
  float gm = -INFINITY, gl = 0.f;
  for (int s = 0; s < splits; ++s) gm = fmaxf(gm, part_ml[(base + s) * 2]);
  for (int s = 0; s < splits; ++s) {
    const float ms = part_ml[(base + s) * 2];
    gl += ms == -INFINITY ? 0.f : part_ml[(base + s) * 2 + 1] * ex2(ms - gm);
  }
  if (p.sink) gl += ex2(p.sink[h] * LOG2E_F - (gm == -INFINITY ? 0.f : gm));
  float f = gl == 0.f ? 0.f : 1.f / gl;
  if (p.gate) f *= p.gate[b * p.H + h];
  for (int c = threadIdx.x * 4; c < p.o_hd; c += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < splits; ++s) {
      const float ms = part_ml[(base + s) * 2];
      if (ms == -INFINITY) continue;
      const float e = ex2(ms - gm);
      const float4 v = *reinterpret_cast<const float4*>(part_o + (base + s) * p.o_hd + c);
      a.x += v.x * e; a.y += v.y * e; a.z += v.z * e; a.w += v.w * e;
    }
    const float r[4] = {a.x * f, a.y * f, a.z * f, a.w * f};
    put_n<bf16, 4>(reinterpret_cast<bf16*>(p.out) + (b * p.H + h) * p.o_hd + c, r);
  }
}

template <typename K>
int allow_smem(K kernel, int bytes, int* have) {
  int dev = 0;
  DLTI_CUDA_CHECK(cudaGetDevice(&dev));
  if (have[dev & 63] < bytes) {
    DLTI_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    have[dev & 63] = bytes;
  }
  return 0;
}

template <int HT, int W16>
int launch_latent(const LatentParams& p, long long rows, int splits, float* ws, cudaStream_t st) {
  static int have[64] = {};
  int stages = LSTAGES;
  while (stages > 2 && LatentSmem<HT>::bytes(p.pitch, stages) > 227 * 1024) --stages;
  const int smem = LatentSmem<HT>::bytes(p.pitch, stages);
  if (smem > 227 * 1024) { dlti_set_error("latent_decode: cache rows too long for shared memory"); return DLTI_ERR_TOO_LARGE; }
  if (int rc = allow_smem(latent_decode_kernel<HT, W16>, smem, have)) return rc;
  float* ml = splits > 1 ? ws + rows * p.H * splits * p.o_hd : nullptr;
  DLTI_CUDA_CHECK(dlti_launch_pdl(rows, latent_decode_kernel<HT, W16>, dim3(splits, (p.H + 16 * HT - 1) / (16 * HT), (unsigned)rows), dim3(LTHREADS),
                                  (size_t)smem, st, p, splits, stages, ws, ml));
  dlti_count_launch();
  if (splits > 1) {
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, latent_combine_kernel, dim3(p.H, (unsigned)rows), dim3(128), 0, st, p, splits, (const float*)ws,
                                    (const float*)ml));
    dlti_count_launch();
  }
  return 0;
}

}  // namespace

// Projection rows -> queries, cache rows at slots (-1: none) and sigmoid gates; rows t < nabs in the absorbed layout, the
// others in the expanded one (see PrepParams).
DLTI_API int dlti_latent_prep(const void* proj, long long ld, int oq, int od, int og, int H, int dim, int rot, int rank, int rd, int interleaved,
                              const float* cos_t, const float* sin_t, const int* pos, const float* kvw, float eps, const long long* slots,
                              void* cache, int pitch, int rot_at, int nabs, void* qn, int qn_hd, void* ql, void* qp, long long qp_ld, int qp_hd,
                              void* lat, const int* qdst, const int* dst, float* gate, long long tokens, int acc, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (H < 1 || dim < 1 || rot < 0 || rank < 1 || rd % 2 || rd > rot || rot_at < rank || pitch < rot_at + rot || pitch % 8 || (rd && (!cos_t || !sin_t)) ||
      (nabs > 0 && (!qn || !ql)) || (nabs < tokens && (!qp || !lat)) || (og >= 0 && !gate)) return DLTI_ERR_BAD_ARG;
  if (acc && dtype != DLTI_BF16) return DLTI_ERR_UNSUPPORTED;
  PrepParams p{proj, ld, oq, od, og, H, dim, rot, rank, rd, interleaved, cos_t, sin_t, pos, kvw, eps, slots, cache, pitch, rot_at,
               nabs, qn, qn_hd, ql, qp, qp_ld, qp_hd, lat, qdst, dst, gate, tokens};
  const uintptr_t al = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(qn) |
                       reinterpret_cast<uintptr_t>(ql) | reinterpret_cast<uintptr_t>(qp) | reinterpret_cast<uintptr_t>(lat) | reinterpret_cast<uintptr_t>(kvw);
  if (dtype == DLTI_BF16 && (interleaved || rd == 0) && dim % 8 == 0 && rot % 8 == 0 && rank % 8 == 0 && rd % 8 == 0 && rank <= 1024 && ld % 8 == 0 &&
      oq % 8 == 0 && od % 8 == 0 && pitch % 8 == 0 && rot_at % 8 == 0 && qn_hd == dim && qp_ld % 8 == 0 && qp_hd % 8 == 0 && (al & 15) == 0 &&
      tokens < (1ll << 31)) {
    const int za = (pitch - rank - rot) / 8, zp = nabs < tokens ? (qp_hd - dim - rot) / 8 : 0;
    const int per_head = (dim + rot) / 8 + (za > zp ? za : zp), units = H * per_head;
    const int qpn = acc ? 1 : 2, per = 128 * qpn;
    auto kern = acc ? latent_prep_vec_kernel<true, 1> : latent_prep_vec_kernel<false, 2>;
    DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, kern, dim3((unsigned)tokens, 1 + (units + per - 1) / per), dim3(128), 0, st, p, units, per_head));
    dlti_count_launch();
    return 0;
  }
  const size_t smem = (size_t)rank * 4;
  if (smem > 47 * 1024) { dlti_set_error("latent_prep: latents of up to 12032 elements"); return DLTI_ERR_TOO_LARGE; }
  if (acc) {
    DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, latent_prep_kernel<bf16, true>, dim3((unsigned)tokens), dim3(128), smem, st, p));
  } else {
    DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(tokens, latent_prep_kernel<T, false>, dim3((unsigned)tokens), dim3(128), smem, st, p)));
  }
  dlti_count_launch();
  return 0;
}

DLTI_API int dlti_latent_rows(void* lat, const void* cache, int pitch, const int* rows, const int* slots, long long n, cudaStream_t st) {
  if (n <= 0) return 0;
  if (pitch % 8) return DLTI_ERR_BAD_ARG;
  const long long total = n * (pitch / 8);
  latent_rows_kernel<<<grid_for(total, 256), 256, 0, st>>>((bf16*)lat, (const bf16*)cache, pitch, rows, slots, total);
  dlti_count_launch();
  return (int)cudaGetLastError();
}

// kn: b is [H * K, N], else [H * N, K] (see HeadGemmParams)
DLTI_API int dlti_head_gemm(const void* a, long long a_ld, int a_hd, const void* b, long long b_ld, void* out, long long o_ld, int o_hd,
                            long long rows, int H, int K, int N, int kn, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (H < 1 || K < 1 || N < 1 || H > 65535) return DLTI_ERR_BAD_ARG;
  HeadGemmParams p{a, a_ld, a_hd, b, b_ld, out, o_ld, o_hd, rows, H, K, N};
  if (dtype == DLTI_BF16 && K % 8 == 0 && N % 8 == 0 && a_ld % 8 == 0 && a_hd % 8 == 0 && b_ld % 8 == 0 && o_ld % 2 == 0 && o_hd % 2 == 0 &&
      rows <= 65535ll * HG_M && ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(out)) & 15) == 0) {
    static int have0[64] = {}, have1[64] = {};
    const int smem = HG_STAGES * HG_STAGE;
    if (int rc = kn ? allow_smem(head_gemm_kernel<true>, smem, have1) : allow_smem(head_gemm_kernel<false>, smem, have0)) return rc;
    DLTI_CUDA_CHECK(dlti_launch_pdl(rows, kn ? head_gemm_kernel<true> : head_gemm_kernel<false>,
                                    dim3((N + HG_N - 1) / HG_N, H, (unsigned)((rows + HG_M - 1) / HG_M)), dim3(128), (size_t)smem, st, p));
    dlti_count_launch();
    return 0;
  }
  if (rows > 65535) { dlti_set_error("head_gemm: up to 65535 rows of unaligned sizes"); return DLTI_ERR_TOO_LARGE; }
  const dim3 g((N + 127) / 128, H, (unsigned)rows);
  if (kn) DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, head_gemm_any_kernel<T, true>, g, dim3(128), 0, st, p)));
  else DISPATCH_T(dtype, DLTI_CUDA_CHECK(dlti_launch_pdl(rows, head_gemm_any_kernel<T, false>, g, dim3(128), 0, st, p)));
  dlti_count_launch();
  return 0;
}

// bf16, rank <= 512. q [rows, H, pitch], out [rows, H, o_hd] with o_hd = round16(rank); heads a CTA: 16 or 32.
// ws: rows * H * splits * (o_hd + 2) floats.
DLTI_API int dlti_latent_decode(const void* q, const void* cache, int pitch, int rank, const int* tables, int max_blocks, int bs, const int* ctx,
                                const int* rseq, const int* pos, long long rows, int H, float scale, const float* sink, const float* gate,
                                int heads_per_cta, int splits, float* ws, void* out, int o_hd, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (H < 1 || rank < 1 || pitch % 16 != 8 || o_hd % 16 || o_hd < rank || o_hd > pitch || splits < 1 || rows > 65535 || (splits > 1 && !ws) ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15)) return DLTI_ERR_BAD_ARG;
  if (rank > 512) { dlti_set_error("latent_decode: latents of up to 512 elements"); return DLTI_ERR_TOO_LARGE; }
  LatentParams p{q, cache, pitch, rank, tables, max_blocks, bs, ctx, rseq, pos, H, scale, sink, gate, out, o_hd};
  const bool two = heads_per_cta > 16;
  if (rank <= 128) return two ? launch_latent<2, 1>(p, rows, splits, ws, st) : launch_latent<1, 1>(p, rows, splits, ws, st);
  if (rank <= 256) return two ? launch_latent<2, 2>(p, rows, splits, ws, st) : launch_latent<1, 2>(p, rows, splits, ws, st);
  return two ? launch_latent<2, 4>(p, rows, splits, ws, st) : launch_latent<1, 4>(p, rows, splits, ws, st);
}

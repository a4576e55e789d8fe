// Attention over the paged cache for the layer-stack models: any head size, grouped key/value heads, causal or chunked
// (position i sees keys of its own chunk of `chunk` positions only), optional per-head output gate.
//
//   attn_rows_kernel     one warp per (row, head), fp32 arithmetic throughout: the fp32 mode
#include "common.cuh"

namespace {

struct PagedParams {
  const void* q; long long q_ld; int q_hd;         // queries: row pitch, head pitch
  const void *kc, *vc; int kd, vd;                 // cache row pitches of a head
  const int* tables; int max_blocks; int bs;
  const int *ctx, *cu, *rseq, *pos; int nd;
  int H, G, dim, vdim, chunk;
  float scale;
  const float* gate;                               // [rows, H] factors or null
  void* out; long long o_ld;                       // head h at column h * vdim
  long long rows;
};

__device__ __forceinline__ int first_key(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

constexpr int ROWS_MAXV = 16;                      // value dims per lane: heads of up to 512
template <typename T>
__global__ void __launch_bounds__(128) attn_rows_kernel(const PagedParams p) {
  extern __shared__ float sq_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sq = sq_all + warp * p.dim;
  const long long w = (long long)blockIdx.x * 4 + warp;
  if (w >= p.rows * p.H) return;
  const long long t = w / p.H;
  const int h = (int)(w - t * p.H), g = h / (p.H / p.G);
  const int seq = p.rseq[t], ps = p.pos[t];
  const int nkeys = min(ps + 1, p.ctx[seq]);       // padding rows of a decode graph have no keys
  const int* tab = p.tables + (long long)seq * p.max_blocks;
  const T* qr = reinterpret_cast<const T*>(p.q) + t * p.q_ld + (long long)h * p.q_hd;
  for (int c = lane; c < p.dim; c += 32) sq[c] = Cvt<T>::to_f(qr[c]);
  __syncwarp();
  float m = -INFINITY, l = 0.f, o[ROWS_MAXV];
#pragma unroll
  for (int i = 0; i < ROWS_MAXV; ++i) o[i] = 0.f;
  for (int j0 = first_key(ps, p.chunk); j0 < nkeys; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    long long slot = 0;
    if (j < nkeys) {
      slot = (long long)tab[j / p.bs] * p.bs + j % p.bs;
      const T* kr = reinterpret_cast<const T*>(p.kc) + (slot * p.G + g) * p.kd;
      float a = 0.f;
      for (int c = 0; c < p.dim; ++c) a = fmaf(sq[c], Cvt<T>::to_f(kr[c]), a);
      s = a * p.scale;
    }
    const float nm = fmaxf(m, warp_max(s));
    const float alpha = expf(m - nm);
    const float pj = expf(s - nm);
    l = l * alpha + warp_sum(pj);
    m = nm;
#pragma unroll
    for (int i = 0; i < ROWS_MAXV; ++i) o[i] *= alpha;
    const int nj = min(32, nkeys - j0);
    for (int jj = 0; jj < nj; ++jj) {
      const float pp = __shfl_sync(0xffffffffu, pj, jj);
      const long long sl = __shfl_sync(0xffffffffu, slot, jj);
      const T* vr = reinterpret_cast<const T*>(p.vc) + (sl * p.G + g) * p.vd;
#pragma unroll
      for (int i = 0; i < ROWS_MAXV; ++i) {
        const int c = lane + 32 * i;
        if (c < p.vdim) o[i] = fmaf(pp, Cvt<T>::to_f(vr[c]), o[i]);
      }
    }
  }
  float f = l > 0.f ? 1.f / l : 0.f;
  if (p.gate) f *= p.gate[t * p.H + h];
  T* orow = reinterpret_cast<T*>(p.out) + t * p.o_ld + (long long)h * p.vdim;
#pragma unroll
  for (int i = 0; i < ROWS_MAXV; ++i) {
    const int c = lane + 32 * i;
    if (c < p.vdim) orow[c] = Cvt<T>::from_f(o[i] * f);
  }
}

template <typename T>
int launch_rows(const PagedParams& p, cudaStream_t st) {
  const size_t smem = (size_t)4 * p.dim * 4;
  attn_rows_kernel<T><<<(unsigned)((p.rows * p.H + 3) / 4), 128, smem, st>>>(p);
  dlti_count_launch();
  return (int)cudaGetLastError();
}

}  // namespace

// rows of decode sequences (row s = sequence s < nd) and of prompts (sequence nd + i: rows nd + cu[i] ... nd + cu[i+1]).
DLTI_API int dlti_attn_rows(const void* q, long long q_ld, int q_hd, const void* kc, const void* vc, int kd, int vd, const int* tables,
                            int max_blocks, int bs, const int* ctx, const int* rseq, const int* pos, int H, int G, int dim, int vdim,
                            int chunk, float scale, const float* gate, void* out, long long o_ld, long long rows, int dtype,
                            cudaStream_t st) {
  if (rows <= 0) return 0;
  if (H % G || dim < 1 || vdim < 1) return DLTI_ERR_BAD_ARG;
  if (dim > 512 || vdim > 512) { dlti_set_error("attn_rows: heads of up to 512 dimensions"); return DLTI_ERR_TOO_LARGE; }
  PagedParams p{q, q_ld, q_hd, kc, vc, kd, vd, tables, max_blocks, bs, ctx, nullptr, rseq, pos, 0, H, G, dim, vdim, chunk, scale,
                gate, out, o_ld, rows};
  if (dtype == DLTI_BF16) return launch_rows<__nv_bfloat16>(p, st);
  if (dtype == DLTI_FP32) return launch_rows<float>(p, st);
  return DLTI_ERR_UNSUPPORTED;
}

// Latent attention, everything but its matrix products, for bf16 and fp32 storage:
//   hy_latent_in     after the input projection: RMS norm of the query latent (if any) in place; the key/value latent
//                    (normed) and the shared rotated key part into the token's page row
//   hy_latent_q      rotation of every head's rotated query part, in place for rows whose keys are multiplied
//                    out, beside the absorbed query for the others
//   hy_latent_gather page rows of prompt portions and the keys before them into one contiguous matrix
//   hy_latent_attn   absorbed attention straight on page rows, one warp per (row, head), any sizes: the fp32
//                    path, and the path of head sizes the tensor-core kernels do not cover
// A page row is (latent | rotated key part): its score with the absorbed query (W_uk^T q | rotated q) is the
// head's whole score, and the weighted sum of its first part is what W_uv turns into the head's output.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int LAT_THREADS = 128;

// Rotation of the pairs (2i, 2i + 1) of 8 consecutive entries: their angles, then the entries.
struct Angles4 {
  float c[4], s[4];
};
__device__ __forceinline__ Angles4 load_angles(const float* ct, const float* st, int d, int rot) {
  Angles4 a;
  if ((rot & 7) == 0) {
    const float4 c = *reinterpret_cast<const float4*>(ct + (d >> 1)), s = *reinterpret_cast<const float4*>(st + (d >> 1));
    return {{c.x, c.y, c.z, c.w}, {s.x, s.y, s.z, s.w}};
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const bool in = d + 2 * j < rot;         // padding is zero and stays so
    a.c[j] = in ? ct[(d >> 1) + j] : 1.f;
    a.s[j] = in ? st[(d >> 1) + j] : 0.f;
  }
  return a;
}
__device__ __forceinline__ void rotate_pairs8(float (&f)[8], const Angles4& a) {
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float u = f[2 * j], v = f[2 * j + 1];
    f[2 * j] = u * a.c[j] - v * a.s[j];
    f[2 * j + 1] = v * a.c[j] + u * a.s[j];
  }
}

// A thread's vectors of the row (query latent, then page row) stay in registers up to KEEP of them.  TPR threads share
// a row: the block, or a warp where rows are short.
template <typename T, int TPR>
__global__ void __launch_bounds__(LAT_THREADS, sizeof(T) == 2 ? 10 : 6)
hy_latent_in_kernel(const __grid_constant__ BbHyLayer L, T* __restrict__ proj, int ld, const int* __restrict__ pos_,
                    const int* __restrict__ row_seq, const int* __restrict__ tables, int max_blocks, int bs, float eps, int rows) {
  constexpr int KEEP = 2;
  __shared__ float buf[2][32];
  const int tid = threadIdx.x % TPR, r = blockIdx.x * (LAT_THREADS / TPR) + threadIdx.x / TPR;
  if (r >= rows) return;
  const int width = L.kvrp + L.rotp, n = L.qrp + (L.own_kv ? width : 0);
  T* q = proj + (size_t)r * ld + L.off_dq;
  const T* c = proj + (size_t)r * ld + L.off_ckv;
  const int pos = pos_[r];
  float v[KEEP][8], gain[8], sq = 0.f, sc = 0.f;
  auto sum = [&](int i, const float (&f)[8]) {
    float t = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) t += f[j] * f[j];
    if (i < L.qrp) sq += t;
    else if (i < L.qrp + L.kvrp) sc += t;
  };
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = (tid + t * TPR) * 8;
    if (i < n) load8(i < L.qrp ? q + i : c + (i - L.qrp), v[t]);
  }
  // the first vector's gains are asked for before the sums are known
  auto gains = [&](int i) { return i < L.qrp ? L.dq_norm + i : L.dkv_norm + (i - L.qrp); };
  if (tid * 8 < min(n, L.qrp + L.kvrp)) load8(gains(tid * 8), gain);
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = (tid + t * TPR) * 8;
    if (i < n) sum(i, v[t]);
  }
  for (int i = (tid + KEEP * TPR) * 8; i < n; i += TPR * 8) {
    float f[8];
    load8(i < L.qrp ? q + i : c + (i - L.qrp), f);
    sum(i, f);
  }
  const int blk = L.own_kv ? tables[(size_t)row_seq[r] * max_blocks + pos / bs] : 0;
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if constexpr (TPR > 32) {
    if ((threadIdx.x & 31) == 0) {
      buf[0][threadIdx.x >> 5] = sq;
      buf[1][threadIdx.x >> 5] = sc;
    }
    __syncthreads();
    sq = sc = 0.f;
#pragma unroll
    for (int i = 0; i < LAT_THREADS / 32; ++i) {
      sq += buf[0][i];
      sc += buf[1][i];
    }
  }
  const float rq = 1.f / sqrtf(sq / (float)max(L.qr, 1) + eps), rc = 1.f / sqrtf(sc / (float)L.kvr + eps);
  T* page = static_cast<T*>(L.kc) + ((size_t)blk * bs + pos % bs) * width;
  auto emit = [&](int i, float (&f)[8], bool first) {
    float g[8];
    if (i < L.qrp + L.kvrp) {
      if (first) {
#pragma unroll
        for (int j = 0; j < 8; ++j) g[j] = gain[j];
      } else {
        load8(gains(i), g);
      }
    }
    if (i < L.qrp) {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= rq * g[j];
      store8(q + i, f);
      return;
    }
    i -= L.qrp;
    if (i < L.kvrp) {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= rc * g[j];
    } else {
      const size_t at = (size_t)pos * (L.rot >> 1);
      rotate_pairs8(f, load_angles(L.cos_t + at, L.sin_t + at, i - L.kvrp, L.rot));
    }
    store8(page + i, f);
  };
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = (tid + t * TPR) * 8;
    if (i < n) emit(i, v[t], t == 0);
  }
  for (int i = (tid + KEEP * TPR) * 8; i < n; i += TPR * 8) {
    float f[8];
    load8(i < L.qrp ? q + i : c + (i - L.qrp), f);
    emit(i, f, false);
  }
}

// Rows below n_in rotate in place inside q; row r of the others writes to qa row r - n_in.  Lanes run over the
// vectors of a head's rotated part, then heads; a thread takes every step-th head.
constexpr int LQ_HEADS = 4;

template <typename T>
__global__ void __launch_bounds__(LAT_THREADS)
hy_latent_q_kernel(const __grid_constant__ BbHyLayer L, T* __restrict__ q, int ldq, T* __restrict__ qa, int ldqa,
                   const int* __restrict__ pos_, int n_in, int step) {
  const unsigned vecs = L.rotp / 8, t = blockIdx.y * blockDim.x + threadIdx.x;
  const int h0 = t / vecs, d = (t - h0 * vecs) * 8, r = blockIdx.x;
  if (h0 >= step) return;
  const int pos = pos_[r];
  T* row = q + (size_t)r * ldq + L.dkp + d;
  float f[LQ_HEADS][8];
#pragma unroll
  for (int i = 0; i < LQ_HEADS; ++i)
    if (h0 + i * step < L.hq) load8(row + (h0 + i * step) * (L.dkp + L.rotp), f[i]);
  const size_t at = (size_t)pos * (L.rot >> 1);
  const Angles4 a = load_angles(L.cos_t + at, L.sin_t + at, d, L.rot);
#pragma unroll
  for (int i = 0; i < LQ_HEADS; ++i) {
    const int h = h0 + i * step;
    if (h >= L.hq) break;
    rotate_pairs8(f[i], a);
    store8(r < n_in ? row + h * (L.dkp + L.rotp) : qa + (size_t)(r - n_in) * ldqa + h * (L.kvrp + L.rotp) + L.kvrp + d, f[i]);
  }
}

__global__ void __launch_bounds__(LAT_THREADS)
hy_latent_gather_kernel(const uint4* __restrict__ pages, const int* __restrict__ src, uint4* __restrict__ out, int vecs,
                        int ld_vecs, int rows, int pool_rows) {
  const unsigned t = blockIdx.x * LAT_THREADS + threadIdx.x;
  const int r = t / (unsigned)vecs, v = t - r * vecs;
  if (r >= rows) return;
  const int p = min(max(src[r], 0), pool_rows - 1);
  out[(size_t)r * ld_vecs + v] = pages[(size_t)p * vecs + v];
}

// V: elements of a lane (page rows up to 32 V wide).  Row r of qa / out is batch row r.
template <typename T, int V>
__global__ void __launch_bounds__(LAT_THREADS)
hy_latent_attn_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ qa, int ldq, T* __restrict__ out, int ldo,
                      const int* __restrict__ pos_, const int* __restrict__ row_seq, const int* __restrict__ tables,
                      int max_blocks, int bs, int rows, const T* __restrict__ gate, int ldg) {
  const int w = (blockIdx.x * LAT_THREADS + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (w >= rows * L.hq) return;
  const int r = w / L.hq, h = w % L.hq, width = L.kvrp + L.rotp;
  const T* q = qa + (size_t)r * ldq + h * width;
  float qf[V], o[V];
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const int d = lane + 32 * i;
    qf[i] = d < width ? to_f(q[d]) * L.scale : 0.f;
    o[i] = 0.f;
  }
  const int last = pos_[r], first = L.window > 0 ? max(0, last - L.window + 1) : 0;
  const int* bt = tables + (size_t)row_seq[r] * max_blocks;
  const T* pages = static_cast<const T*>(L.kc);
  float m = -INFINITY, l = 0.f;
  for (int j = first; j <= last; ++j) {
    const T* row = pages + ((size_t)bt[j / bs] * bs + j % bs) * width;
    float k[V], s = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const int d = lane + 32 * i;
      k[i] = d < width ? to_f(row[d]) : 0.f;
      s = fmaf(qf[i], k[i], s);
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s);
    const float al = expf(m - mn), p = expf(s - mn);
    l = fmaf(l, al, p);
    m = mn;
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] = fmaf(p, k[i], o[i] * al);
  }
  float f = 1.f / l;
  if (gate) f *= sigmoid_f(to_f(gate[(size_t)r * ldg + h]));
  T* dst = out + (size_t)r * ldo + h * L.kvrp;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const int d = lane + 32 * i;
    if (d < L.kvrp) dst[d] = from_f<T>(o[i] * f);
  }
}

template <typename T>
static int launch_attn(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, int bs, int r0, int r1,
                       cudaStream_t s) {
  const int rows = r1 - r0, width = L.kvrp + L.rotp;
  const T* gate = L.gate_kind == 1 ? static_cast<const T*>(w.proj) + (size_t)r0 * w.ld_proj + L.off_g : nullptr;
  const int grid = (int)(((long)rows * L.hq * 32 + LAT_THREADS - 1) / LAT_THREADS);
#define BB_LAUNCH_LA(V)                                                                                            \
  hy_latent_attn_kernel<T, V><<<grid, LAT_THREADS, 0, s>>>(L, static_cast<const T*>(w.qa), w.ld_qa,                \
                                                           static_cast<T*>(w.ol), w.ld_ol, b.pos + r0,             \
                                                           b.row_seq + r0, b.tables, b.max_blocks, bs, rows, gate, \
                                                           w.ld_proj)
  if (width <= 128) BB_LAUNCH_LA(4);
  else if (width <= 256) BB_LAUNCH_LA(8);
  else if (width <= 640) BB_LAUNCH_LA(20);
  else if (width <= 1280) BB_LAUNCH_LA(40);
  else return BB_ESIZE;
#undef BB_LAUNCH_LA
  return (int)cudaGetLastError();
}

}  // namespace bb

using namespace bb;

BB_API int bb_hy_latent_in(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  cudaStream_t s = (cudaStream_t)stream;
  const bool small = L->qrp + (L->own_kv ? L->kvrp + L->rotp : 0) <= 2 * 32 * 8;
  const int grid = small ? (b->n + LAT_THREADS / 32 - 1) / (LAT_THREADS / 32) : b->n;
#define BB_LAT_IN(T, TPR)                                                                                                    \
  hy_latent_in_kernel<T, TPR><<<grid, LAT_THREADS, 0, s>>>(*L, static_cast<T*>(w->proj), w->ld_proj, b->pos, b->row_seq,     \
                                                           b->tables, b->max_blocks, c->block_size, c->eps, b->n)
  if (c->dtype) {
    if (small) BB_LAT_IN(float, 32);
    else BB_LAT_IN(float, LAT_THREADS);
  } else {
    if (small) BB_LAT_IN(__nv_bfloat16, 32);
    else BB_LAT_IN(__nv_bfloat16, LAT_THREADS);
  }
#undef BB_LAT_IN
  return (int)cudaGetLastError();
}

// n_in: leading rows whose rotated queries stay in place.
BB_API int bb_hy_latent_q(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int n_in, void* stream) {
  cudaStream_t s = (cudaStream_t)stream;
  const int step = (L->hq + LQ_HEADS - 1) / LQ_HEADS;
  const int lanes = step * (L->rotp / 8), t = lanes < LAT_THREADS ? (lanes + 31) & ~31 : LAT_THREADS;
  const dim3 grid(b->n, (lanes + t - 1) / t);
  int ldq;
  void* q = hy_latent_queries(*c, *L, *w, &ldq);
  if (c->dtype)
    hy_latent_q_kernel<float><<<grid, t, 0, s>>>(*L, static_cast<float*>(q), ldq, static_cast<float*>(w->qa), w->ld_qa, b->pos,
                                                 n_in, step);
  else
    hy_latent_q_kernel<__nv_bfloat16><<<grid, t, 0, s>>>(*L, static_cast<__nv_bfloat16*>(q), ldq,
                                                         static_cast<__nv_bfloat16*>(w->qa), w->ld_qa, b->pos, n_in, step);
  return (int)cudaGetLastError();
}

BB_API int bb_hy_latent_gather(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->n_exp <= 0) return BB_OK;
  if (c->dtype || b->n_exp > w->exp_rows) return BB_EARG;
  const int vecs = (L->kvrp + L->rotp) / 8;
  const long t = (long)b->n_exp * vecs;
  hy_latent_gather_kernel<<<(int)((t + LAT_THREADS - 1) / LAT_THREADS), LAT_THREADS, 0, (cudaStream_t)stream>>>(
      static_cast<const uint4*>(L->kc), b->exp_src, static_cast<uint4*>(w->ckv), vecs, w->ld_ckv / 8, b->n_exp,
      w->pool_blocks * c->block_size);
  return (int)cudaGetLastError();
}

// Absorbed attention of batch rows r0 .. r1 - 1 (rows 0 .. of w->qa and w->ol).
BB_API int bb_hy_latent_attn(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int r0, int r1,
                             void* stream) {
  if (r0 >= r1) return BB_OK;
  return c->dtype ? launch_attn<float>(*L, *w, *b, c->block_size, r0, r1, (cudaStream_t)stream)
                  : launch_attn<__nv_bfloat16>(*L, *w, *b, c->block_size, r0, r1, (cudaStream_t)stream);
}

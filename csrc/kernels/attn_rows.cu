// Attention of single query rows against the paged K/V pool, one warp per (row, query head): any head
// sizes up to 512, bf16 or fp32 pages, soft-capped scores, windows, means of blocks behind them, sinks, output gates (per
// head or per element), outputs turned back.  It is the fp32 path and the path of head sizes the tensor-core prefill and
// the split-KV decode kernels do not cover.
#include "../common/host.hpp"
#include "../common/pooled.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"

namespace bb {

// AR_VEC: elements of a lane (head sizes up to 32 times that)
template <typename T, int AR_VEC>
__global__ void __launch_bounds__(128)
attn_rows_kernel(const T* __restrict__ q, int ldq, const T* __restrict__ kc, const T* __restrict__ vc,
                 const int* __restrict__ pos, const int* __restrict__ row_seq, const int* __restrict__ tables,
                 int max_blocks, int bs, T* __restrict__ out, int ldo, const T* __restrict__ gate, int ldg, int rows,
                 int hq, int hk, int dk, int dv, int dkp, int dvp, float scale, float softcap, int gate_elems, float out_scale,
                 int window, const BbPooled x) {
  const int w = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (w >= rows * hq) return;
  const int r = w / hq, h = w % hq, g = h / (hq / hk);
  float qf[AR_VEC], o[AR_VEC];
#pragma unroll
  for (int i = 0; i < AR_VEC; ++i) {
    const int d = lane + 32 * i;
    qf[i] = d < dk ? to_f(q[(size_t)r * ldq + h * dkp + d]) * scale : 0.f;
    o[i] = 0.f;
  }
  const int last = pos[r];
  const int* bt = tables + (size_t)row_seq[r] * max_blocks;
  float m = -INFINITY, l = 0.f;
  const int first = window > 0 ? max(last - window + 1, 0) : 0, means = x.pool > 0 ? first / x.pool : 0;
  for (int j = first - means; j <= last; ++j) {
    const T *kp = kc, *vp = vc;
    size_t row;
    if (j < first) {
      const int e = (j - (first - means) + 1) * x.pool - 1;      // last token of the block
      row = ((size_t)bt[e / bs] * hk + g) * x.pool_rows + e % bs / x.pool;
      kp = static_cast<const T*>(x.pkc);
      vp = static_cast<const T*>(x.pvc);
    } else {
      row = ((size_t)bt[j / bs] * hk + g) * bs + j % bs;
    }
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < AR_VEC; ++i) {
      const int d = lane + 32 * i;
      if (d < dk) s = fmaf(qf[i], to_f(kp[row * dkp + d]), s);
    }
    s = warp_sum(s);
    if (softcap > 0.f) s = softcap * tanhf(s / softcap);
    const float mn = fmaxf(m, s);
    const float al = expf(m - mn), p = expf(s - mn);
    l = l * al + p;
    m = mn;
#pragma unroll
    for (int i = 0; i < AR_VEC; ++i) {
      const int d = lane + 32 * i;
      if (d < dv) o[i] = fmaf(p, to_f(vp[row * dvp + d]), o[i] * al);
    }
  }
  if (x.sink) {             // (against the maximum of both, so that neither exponential overflows)
    const float sk = x.sink[h], mn = fmaxf(m, sk), al = expf(m - mn);
    l = l * al + expf(sk - mn);
#pragma unroll
    for (int i = 0; i < AR_VEC; ++i) o[i] *= al;
  }
  if (x.vcos) {
    const int half = x.vturn >> 1;
#pragma unroll
    for (int i = 0; i < AR_VEC; ++i) {
      const int d = lane + 32 * i;
      const size_t t = (size_t)last * half + min(d >> 1, half - 1);
      const float other = __shfl_xor_sync(0xffffffffu, o[i], 1), co = x.vcos[t], si = x.vsin[t];
      o[i] = fmaf(o[i], co, d & 1 ? -other * si : other * si);
    }
  }
  float f = out_scale / l;
  if (gate && !gate_elems) f *= sigmoid_f(to_f(gate[(size_t)r * ldg + h]));
#pragma unroll
  for (int i = 0; i < AR_VEC; ++i) {
    const int d = lane + 32 * i;
    if (d >= dvp) continue;
    float v = d < dv ? o[i] * f : 0.f;
    if (gate && gate_elems) v *= sigmoid_f(to_f(gate[(size_t)r * ldg + h * dvp + d]));
    out[(size_t)r * ldo + h * dvp + d] = from_f<T>(v);
  }
}

}  // namespace bb

// dtype 0 bf16, 1 fp32.  Row r attends keys [0, pos[r]] of sequence row_seq[r]; head h of q at column
// h dkp, of out at column h dvp; gate (may be null): raw gate values, head h at column h, or with gate_elems one for
// every output column.  window: the latest keys of a row, itself included (0: all); xt (may be null): what lies behind it,
// sinks and rotated values.
BB_API int bb_attn_rows_p(int dtype, const void* q, int ldq, const void* kc, const void* vc, const int* pos,
                        const int* row_seq, const int* tables, int max_blocks, int bs, void* out, int ldo,
                        const void* gate, int ldg, int rows, int hq, int hk, int dk, int dv, int dkp, int dvp,
                          float scale, float softcap, int gate_elems, float out_scale, int window, const BbPooled* xt,
                          void* stream) {
  using namespace bb;
  if (rows <= 0) return BB_OK;
  const int d = dk > dvp ? dk : dvp;
  if (d > 512 || hq % hk) return BB_ESIZE;
  const BbPooled x = xt ? *xt : BbPooled{};
  if (x.pool > 0 && (window <= 0 || x.pool_rows * x.pool < bs)) return BB_EARG;
  const int grid = (int)(((long)rows * hq * 32 + 127) / 128);
  cudaStream_t s = (cudaStream_t)stream;
#define BB_LAUNCH_AR(T, V)                                                                                          \
  attn_rows_kernel<T, V><<<grid, 128, 0, s>>>((const T*)q, ldq, (const T*)kc, (const T*)vc, pos, row_seq, tables,   \
                                              max_blocks, bs, (T*)out, ldo, (const T*)gate, ldg, rows, hq, hk, dk,  \
                                              dv, dkp, dvp, scale, softcap, gate_elems, out_scale, window, x)
#define BB_LAUNCH_AR_T(T)                  \
  do {                                     \
    if (d <= 64) BB_LAUNCH_AR(T, 2);       \
    else if (d <= 128) BB_LAUNCH_AR(T, 4); \
    else if (d <= 256) BB_LAUNCH_AR(T, 8); \
    else BB_LAUNCH_AR(T, 16);              \
  } while (0)
  if (dtype) BB_LAUNCH_AR_T(float);
  else BB_LAUNCH_AR_T(__nv_bfloat16);
#undef BB_LAUNCH_AR_T
#undef BB_LAUNCH_AR
  return (int)cudaGetLastError();
}

BB_API int bb_attn_rows(int dtype, const void* q, int ldq, const void* kc, const void* vc, const int* pos,
                        const int* row_seq, const int* tables, int max_blocks, int bs, void* out, int ldo,
                        const void* gate, int ldg, int rows, int hq, int hk, int dk, int dv, int dkp, int dvp,
                        float scale, float softcap, int gate_elems, float out_scale, int window, void* stream) {
  return bb_attn_rows_p(dtype, q, ldq, kc, vc, pos, row_seq, tables, max_blocks, bs, out, ldo, gate, ldg, rows, hq, hk, dk, dv,
                        dkp, dvp, scale, softcap, gate_elems, out_scale, window, nullptr, stream);
}

// Native forward of the hybrid decoder: one host call issues every kernel of a step over one packed
// batch (prompt portions of several sequences and single decoded tokens together), from the embedding
// to the logits of the rows that are asked for.  A layer is
//   residual -> RMS norm -> ONE projection GEMM (mixer inputs, gates and feed-forward halves stacked)
//   -> mixer (attention over the pages, or the state-space recurrence over the slots)
//   -> ONE output GEMM over (mixer output | feed-forward product), scaled and added into the fp32
//      residual stream by its epilogue.
// bf16: the tensor-core GEMM, paged flash prefill, split-KV decode attention and chunked state-space
// kernels; fp32: the CUDA-core forms of the same steps.
#include <cstdint>

#include "../common/host.hpp"
#include "hybrid.hpp"

using namespace bb;

extern "C" {
int bb_gemm_bf16(const void* A, const void* B, void* C, const float* bias, int M, int N, int K, int lda, int ldb, int ldc,
                 int a_mn, int b_mn, int out_mode, float alpha, int bn, int max_ctas, void* stream);
int bb_sgemm(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc, float alpha,
             int accumulate, void* stream);
int bb_hy_embed_norm(const BbHyCfg* c, const int* tok, float* x, int n, void* stream);
int bb_hy_norm(int dtype, const float* x, const int* rows, const float* w, void* h, int n, int d, int dp, float eps,
               void* stream);
int bb_hy_attn_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_mamba_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_conv(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_ssm_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_ssd_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_ssm_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_attn_rows(int dtype, const void* q, int ldq, const void* kc, const void* vc, const int* pos, const int* row_seq,
                 const int* tables, int max_blocks, int bs, void* out, int ldo, const void* gate, int ldg, int rows, int hq,
                 int hk, int dk, int dv, int dkp, int dvp, float scale, float softcap, void* stream);
int bb_flash_fwd_paged_x(const void* q, int ldq, const void* k_pool, const void* v_pool, void* out, int ldo,
                         const int* block_tables, int max_blocks, int block_rows, int pool_blocks, const int* seq_row0,
                         const int* seq_ctx, const int* tile_seq, const int* tile_qt, int n_tiles, int total_rows, int hq,
                         int hk, int dq, int dv, float scale, float softcap, const void* gate, int ldg, void* stream);
int bb_paged_decode_x(const void* q, int ldq, const void* kc, const void* vc, const int* block_tables, int max_blocks,
                      const int* seqlens, void* out, int ldo, float* part_o, float* part_ml, int B, int hq, int hk, int dk,
                      int dv, int bs, int splits, float scale, float softcap, const void* gate, int ldg, void* stream);
}

namespace {

#define BB_TRY(expr)          \
  do {                        \
    int rc_ = (expr);         \
    if (rc_ != 0) return rc_; \
  } while (0)

// y = x W^T
int project(const BbHyCfg& c, const BbHyLin& L, const void* x, int ldx, void* y, int ldy, int rows, void* s) {
  if (c.dtype)
    return bb_sgemm(static_cast<const float*>(x), static_cast<const float*>(L.w), static_cast<float*>(y), rows, L.n, L.k,
                    ldx, L.k, ldy, 1.f, 0, s);
  return bb_gemm_bf16(x, L.w, y, nullptr, rows, L.n, L.k, ldx, L.k, ldy, 0, 0, 0, 1.f, 0, 0, s);
}

// fp32 y (+)= alpha x W^T
int project_f32(const BbHyCfg& c, const BbHyLin& L, const void* x, int ldx, float* y, int ldy, int rows, float alpha,
                int add, void* s) {
  if (c.dtype)
    return bb_sgemm(static_cast<const float*>(x), static_cast<const float*>(L.w), y, rows, L.n, L.k, ldx, L.k, ldy, alpha,
                    add, s);
  return bb_gemm_bf16(x, L.w, y, nullptr, rows, L.n, L.k, ldx, L.k, ldy, 0, 0, add ? 2 : 1, alpha, 0, 0, s);
}

const void* at(const BbHyCfg& c, const void* p, size_t elems) {
  return static_cast<const char*>(p) + elems * (c.dtype ? 4 : 2);
}
void* at(const BbHyCfg& c, void* p, size_t elems) { return static_cast<char*>(p) + elems * (c.dtype ? 4 : 2); }

int attention(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  BB_TRY(bb_hy_attn_post(&c, &L, &w, &b, s));
  const void* q = at(c, w.proj, L.off_q);
  const void* gate = at(c, w.proj, L.off_g);
  const int n_dec = b.n - b.n_pre;
  if (b.n_pre > 0) {
    int rc = BB_ESIZE;
    if (!c.dtype)
      rc = bb_flash_fwd_paged_x(q, w.ld_proj, L.kc, L.vc, w.cat, w.ld_cat, b.tables, b.max_blocks, c.block_size,
                                w.pool_blocks, b.seq_row0, b.seq_ctx, b.tile_seq, b.tile_qt, b.n_tiles, b.n_pre, L.hq, L.hk,
                                L.dkp, L.dvp, L.scale, L.softcap, gate, w.ld_proj, s);
    if (rc == BB_ESIZE)
      rc = bb_attn_rows(c.dtype, q, w.ld_proj, L.kc, L.vc, b.pos, b.row_seq, b.tables, b.max_blocks, c.block_size, w.cat,
                        w.ld_cat, gate, w.ld_proj, b.n_pre, L.hq, L.hk, L.dk, L.dv, L.dkp, L.dvp, L.scale, L.softcap, s);
    if (rc) return rc;
  }
  if (n_dec > 0) {
    const void* qd = at(c, q, (size_t)b.n_pre * w.ld_proj);
    const void* gd = at(c, gate, (size_t)b.n_pre * w.ld_proj);
    void* od = at(c, w.cat, (size_t)b.n_pre * w.ld_cat);
    int rc = BB_ESIZE;
    if (!c.dtype) {
      // K/V splits: enough blocks to fill the machine, at most what the partial buffers were sized for
      const int base = n_dec * L.hk;
      int splits = (4 * sm_count() + base - 1) / base;
      splits = splits < 1 ? 1 : (splits > w.splits ? w.splits : splits);
      rc = bb_paged_decode_x(qd, w.ld_proj, L.kc, L.vc, b.tables + (size_t)b.ns_pre * b.max_blocks, b.max_blocks,
                             b.seq_ctx + b.ns_pre, od, w.ld_cat, w.part_o, w.part_ml, n_dec, L.hq, L.hk, L.dkp, L.dvp,
                             c.block_size, splits, L.scale, L.softcap, gd, w.ld_proj, s);
    }
    if (rc == BB_ESIZE)
      rc = bb_attn_rows(c.dtype, qd, w.ld_proj, L.kc, L.vc, b.pos + b.n_pre, b.row_seq + b.n_pre, b.tables, b.max_blocks,
                        c.block_size, od, w.ld_cat, gd, w.ld_proj, n_dec, L.hq, L.hk, L.dk, L.dv, L.dkp, L.dvp, L.scale,
                        L.softcap, s);
    if (rc) return rc;
  }
  return BB_OK;
}

int mamba2(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  if (b.n_pre > 0) {
    BB_TRY(bb_hy_conv(&c, &L, &w, &b, s));
    const int rc = bb_ssd_chunk(&c, &L, &w, &b, s);
    if (rc == BB_ESIZE) BB_TRY(bb_hy_ssm_scan(&c, &L, &w, &b, s));   // fp32, or sizes the tiles do not cover
    else if (rc) return rc;
  }
  BB_TRY(bb_hy_ssm_decode(&c, &L, &w, &b, s));
  return bb_hy_mamba_post(&c, &L, &w, &b, s);
}

}  // namespace

// One step.  Logits land in w->logits [n_want, vocabp]; `trace` (may be null): fp32 [n_layers][n][dp]
// copies of the residual stream after every layer.
BB_API int bb_hybrid_forward(const BbHyCfg* c, const BbHyWork* w, const BbHyBatch* b, float* trace, void* stream) {
  if (!c || !w || !b || b->n <= 0 || b->n > w->rows || b->n_want > w->want_rows) return BB_EARG;
  BB_TRY(bb_hy_embed_norm(c, b->tok, w->x, b->n, stream));
  for (int li = 0; li < c->n_layers; ++li) {
    const BbHyLayer& L = c->layers[li];
    BB_TRY(bb_hy_norm(c->dtype, w->x, nullptr, L.norm, w->h, b->n, c->width, c->dp, c->eps, stream));
    BB_TRY(project(*c, L.in, w->h, c->dp, w->proj, w->ld_proj, b->n, stream));
    BB_TRY(L.kind ? mamba2(*c, L, *w, *b, stream) : attention(*c, L, *w, *b, stream));
    BB_TRY(project_f32(*c, L.out, w->cat, w->ld_cat, w->x, c->dp, b->n, c->residual_mult, 1, stream));
    if (trace) {
      const size_t n = (size_t)b->n * c->dp;
      const cudaError_t e = cudaMemcpyAsync(trace + li * n, w->x, n * 4, cudaMemcpyDeviceToDevice, (cudaStream_t)stream);
      if (e != cudaSuccess) return (int)e;
    }
  }
  if (b->n_want <= 0) return BB_OK;
  BB_TRY(bb_hy_norm(c->dtype, w->x, b->want, c->final_norm, w->hn, b->n_want, c->width, c->dp, c->eps, stream));
  const BbHyLin head{c->head, c->vocabp, c->dp};
  return project_f32(*c, head, w->hn, c->dp, w->logits, c->vocabp, b->n_want, 1.f, 0, stream);
}

// Sizes of the shared structures, for the binding's check of its mirrors.
BB_API int bb_hybrid_sizes(int* out) {
  out[0] = sizeof(BbHyLayer);
  out[1] = sizeof(BbHyCfg);
  out[2] = sizeof(BbHyBatch);
  out[3] = sizeof(BbHyWork);
  return BB_OK;
}

// Native forward of the hybrid decoder: one host call issues every kernel of a step over one packed
// batch (prompt portions of several sequences and single decoded tokens together), from the embedding
// to the logits of the rows that are asked for.  A layer is
//   residual -> RMS norm -> ONE projection GEMM (mixer inputs, gates and feed-forward halves stacked)
//   -> mixer (attention over the pages, or the state-space recurrence over the slots)
//   -> ONE output GEMM over (mixer output | feed-forward product), scaled and added into the fp32
//      residual stream by its epilogue.
// Designs with learned positions or routed experts start their layers in one kernel (hy_start): residual row, plus
// the experts' outputs of the layer before, normed.  A layer may have two mixers side by side, and fp32 products of
// its normed input (router logits, gates of a recurrence) beside the projection GEMM.
// Designs with depth averages keep every layer's result: a layer starts from the weighted sum of all of them
// (written where its own result will be, so the output GEMM adds in place), and its feed-forward has a norm
// and a GEMM of its own.
// Designs with several residual streams run mixer and feed-forward one after the other; between any two of these one
// kernel (hy_streams) spreads the result over the streams and makes the next input.
// bf16: the tensor-core GEMM, paged flash prefill, split-KV decode attention and chunked state-space
// kernels; fp32: the CUDA-core forms of the same steps.
#include <cstdint>
#include <mutex>

#include "../common/host.hpp"
#include "../common/pooled.hpp"
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
int bb_hy_conv_linear(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_mix_norm(const BbHyCfg* c, int li, const BbHyWork* w, const BbHyBatch* b, float* trace, void* stream);
int bb_hy_polynorm(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_latent_in(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_latent_q(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int n_in, void* stream);
int bb_hy_latent_gather(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_latent_attn(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int r0, int r1,
                      void* stream);
int bb_hy_latent_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int qa_row0, void* stream);
int bb_hy_delta_tanh(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_delta(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_rglru(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_gemm_bf16_groups(const void* A, const void* B, void* C, int M, int N, int K, int groups, int lda, int a_step, int ldc,
                        int c_step, void* stream);
int bb_sgemm_groups(const float* A, const float* B, float* C, int M, int N, int K, int groups, int lda, int a_step, int ldc,
                    int c_step, void* stream);
int bb_flash_fwd_window(const void* q, int ldq, const void* k, const void* v, int ldkv, int kv_rows, void* out, int ldo,
                        const int* seq_row0, const int* kv_row0, const int* kv_pos0, const int* seq_ctx, const int* tile_seq,
                        const int* tile_qt, int n_tiles, int total_rows, int hq, int hk, int dq, int dv, float scale,
                        int window, const void* gate, int ldg, void* stream);
int bb_attn_rows_p(int dtype, const void* q, int ldq, const void* kc, const void* vc, const int* pos, const int* row_seq,
                   const int* tables, int max_blocks, int bs, void* out, int ldo, const void* gate, int ldg, int rows, int hq,
                   int hk, int dk, int dv, int dkp, int dvp, float scale, float softcap, int gate_elems, float out_scale,
                   int window, const BbPooled* x, void* stream);
int bb_flash_fwd_paged_p(const void* q, int ldq, const void* k_pool, const void* v_pool, void* out, int ldo,
                         const int* block_tables, int max_blocks, int block_rows, int pool_blocks, const int* seq_row0,
                         const int* seq_ctx, const int* tile_seq, const int* tile_qt, int n_tiles, int total_rows, int hq,
                         int hk, int dq, int dv, float scale, float softcap, const void* gate, int ldg, int gate_elems,
                         float out_scale, int window, const BbPooled* x, void* stream);
int bb_paged_decode_p(const void* q, int ldq, const void* kc, const void* vc, const int* block_tables, int max_blocks,
                      const int* seqlens, void* out, int ldo, float* part_o, float* part_ml, int B, int hq, int hk, int dk,
                      int dv, int bs, int splits, float scale, float softcap, const void* gate, int ldg, int gate_elems,
                      float out_scale, int window, const BbPooled* x, void* stream);
int bb_hy_heads(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_turn(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_pool(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int gather, void* stream);
int bb_hy_streams(const BbHyCfg* c, const BbHyLayer* before, int fq, const BbHyLayer* next, int tq, const BbHyWork* w,
                  const BbHyBatch* b, int all, float* trace, void* stream);
int bb_hy_shift(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_gelu(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_cap(const BbHyCfg* c, const BbHyWork* w, int n, void* stream);
int bb_gla_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_linear_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int marked, void* stream);
int bb_hy_linear_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_linear_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int rows, void* stream);
int bb_retention_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_start(const BbHyCfg* c, int li, const BbHyWork* w, const BbHyBatch* b, int all, float* trace, void* stream);
int bb_hy_kv_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_glu(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_moe_tiles(const BbHyLayer* L, int n);
int bb_hy_route(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_route_row(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_expert_rows(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_expert_glu(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_mlstm_gates(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream);
int bb_hy_mlstm_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int seq0, int n_seq,
                     void* stream);
int bb_hy_mlstm_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_mlstm_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream);
int bb_hy_head_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int rows, void* stream);
int bb_gemm_bf16_grouped(const void* A, const void* B, void* C, int M, int N, int K, int lda, int ldb, int ldc, int b_mn,
                         int out_mode, int group_mode, const int* tile_group, int b_group_rows, int b_total_rows,
                         const int* group_offsets, int num_groups, long c_group_stride, int bn, void* stream);
int bb_sgemm_tiles(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldc, const int* tile_group,
                   void* stream);
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

// y_g = x_g W_g^T for column ranges x_g of x and y_g of y, `xs` and `ys` elements apart; W [groups][n][k]
int project_groups(const BbHyCfg& c, const void* w, int groups, int n, int k, const void* x, int ldx, int xs, void* y, int ldy,
                   int ys, int rows, void* s) {
  if (rows <= 0) return BB_OK;
  if (c.dtype)
    return bb_sgemm_groups(static_cast<const float*>(x), static_cast<const float*>(w), static_cast<float*>(y), rows, n, k,
                           groups, ldx, xs, ldy, ys, s);
  return bb_gemm_bf16_groups(x, w, y, rows, n, k, groups, ldx, xs, ldy, ys, s);
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
  if (L.head_norm) BB_TRY(bb_hy_heads(&c, &L, &w, &b, s));
  else if (L.q_norm) BB_TRY(bb_hy_attn_post(&c, &L, &w, &b, s));
  else BB_TRY(bb_hy_kv_post(&c, &L, &w, &b, s));
  const void* q = at(c, w.proj, L.off_q);
  const void* gate = L.gate_kind ? at(c, w.proj, L.off_g) : nullptr;
  const int elems = L.gate_kind == 2;
  const int n_dec = b.n - b.n_pre;
  const BbPooled x{L.pool, L.pool_rows, L.pkc, L.pvc, w.pk, w.ld_pk, w.pk_rows, b.ctx_row0, L.sink, L.vcos_t, L.vsin_t, L.dv};
  if (b.n_pre > 0) {
    BB_TRY(bb_hy_pool(&c, &L, &w, &b, !c.dtype && L.dkp <= 128 && L.dvp <= 128, s));
    int rc = BB_ESIZE;
    if (!c.dtype)
      rc = bb_flash_fwd_paged_p(q, w.ld_proj, L.kc, L.vc, w.cat, w.ld_cat, b.tables, b.max_blocks, c.block_size,
                                w.pool_blocks, b.seq_row0, b.seq_ctx, b.tile_seq, b.tile_qt, b.n_tiles, b.n_pre, L.hq, L.hk,
                                L.dkp, L.dvp, L.scale, L.softcap, gate, w.ld_proj, elems, L.out_scale, L.window, &x, s);
    if (rc == BB_ESIZE)
      rc = bb_attn_rows_p(c.dtype, q, w.ld_proj, L.kc, L.vc, b.pos, b.row_seq, b.tables, b.max_blocks, c.block_size, w.cat,
                        w.ld_cat, gate, w.ld_proj, b.n_pre, L.hq, L.hk, L.dk, L.dv, L.dkp, L.dvp, L.scale, L.softcap, elems,
                          L.out_scale, L.window, &x, s);
    if (rc) return rc;
  }
  if (n_dec > 0) {
    const void* qd = at(c, q, (size_t)b.n_pre * w.ld_proj);
    const void* gd = gate ? at(c, gate, (size_t)b.n_pre * w.ld_proj) : nullptr;
    void* od = at(c, w.cat, (size_t)b.n_pre * w.ld_cat);
    int rc = BB_ESIZE;
    if (!c.dtype) {
      // K/V splits: enough blocks to fill the machine, at most what the partial buffers were sized for
      const int base = n_dec * L.hk;
      int splits = (4 * sm_count() + base - 1) / base;
      const int keys = L.window + (L.pool > 0 ? b.max_blocks * c.block_size / L.pool : 0);
      if (L.window > 0 && splits > (keys + 31) / 32) splits = (keys + 31) / 32;
      splits = splits < 1 ? 1 : (splits > w.splits ? w.splits : splits);
      rc = bb_paged_decode_p(qd, w.ld_proj, L.kc, L.vc, b.tables + (size_t)b.ns_pre * b.max_blocks, b.max_blocks,
                             b.seq_ctx + b.ns_pre, od, w.ld_cat, w.part_o, w.part_ml, n_dec, L.hq, L.hk, L.dkp, L.dvp,
                             c.block_size, splits, L.scale, L.softcap, gd, w.ld_proj, elems, L.out_scale, L.window, &x, s);
    }
    if (rc == BB_ESIZE)
      rc = bb_attn_rows_p(c.dtype, qd, w.ld_proj, L.kc, L.vc, b.pos + b.n_pre, b.row_seq + b.n_pre, b.tables, b.max_blocks,
                        c.block_size, od, w.ld_cat, gd, w.ld_proj, n_dec, L.hq, L.hk, L.dk, L.dv, L.dkp, L.dvp, L.scale,
                          L.softcap, elems, L.out_scale, L.window, &x, s);
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

// Prompt portions in bf16: keys and values of the window's page rows are multiplied out and the flash kernel
// runs over them; decoded rows (and every row where that kernel does not reach): queries go into the latents'
// space and attention runs on the page rows themselves.
int latent_attention(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  const int dq = L.dkp + L.rotp, width = L.kvrp + L.rotp;
  const int n_in = L.expand.w ? b.n_pre : 0;
  BB_TRY(bb_hy_latent_in(&c, &L, &w, &b, s));
  if (L.uq.w) BB_TRY(project(c, L.uq, at(c, w.proj, L.off_dq), w.ld_proj, w.q, w.ld_q, b.n, s));
  int ldq;
  void* q = hy_latent_queries(c, L, w, &ldq);
  BB_TRY(bb_hy_latent_q(&c, &L, &w, &b, n_in, s));
  if (n_in > 0) {
    BB_TRY(bb_hy_latent_gather(&c, &L, &w, &b, s));
    BB_TRY(project(c, L.expand, w.ckv, w.ld_ckv, w.kvx, w.ld_kvx, b.n_exp, s));
    BB_TRY(bb_flash_fwd_window(q, ldq, w.kvx, at(c, w.kvx, (size_t)L.hq * dq), w.ld_kvx, b.n_exp, w.cat, w.ld_cat,
                               b.seq_row0, b.kv_row0, b.kv_pos0, b.seq_ctx, b.tile_seq, b.tile_qt, b.n_tiles, b.n_pre, L.hq,
                               L.hq, dq, L.dvp, L.scale, L.window, L.gate_kind == 1 ? at(c, w.proj, L.off_g) : nullptr, w.ld_proj, s));
  }
  const int rows = b.n - n_in;
  BB_TRY(project_groups(c, L.w_abs, L.hq, L.kvrp, L.dkp, at(c, q, (size_t)n_in * ldq), ldq, dq, w.qa, w.ld_qa, width, rows, s));
  const int rc = bb_hy_latent_decode(&c, &L, &w, &b, b.n_pre - n_in, s);
  if (rc == BB_OK && n_in < b.n_pre) BB_TRY(bb_hy_latent_attn(&c, &L, &w, &b, n_in, b.n_pre, s));
  else if (rc == BB_ESIZE) BB_TRY(bb_hy_latent_attn(&c, &L, &w, &b, n_in, b.n, s));
  else if (rc) return rc;
  return project_groups(c, L.w_uv, L.hq, L.dvp, L.kvrp, w.ol, w.ld_ol, L.kvrp, at(c, w.cat, (size_t)n_in * w.ld_cat), w.ld_cat,
                        L.dvp, rows, s);
}

int general_delta(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  BB_TRY(bb_hy_delta_tanh(&c, &L, &w, &b, s));
  BB_TRY(project(c, L.w2, at(c, w.proj, L.off_w1), w.ld_proj, w.aux, w.ld_aux, b.n, s));
  return bb_hy_delta(&c, &L, &w, &b, s);
}

int rglru(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  BB_TRY(bb_hy_conv_linear(&c, &L, &w, &b, s));
  BB_TRY(project_groups(c, L.w_gate, L.blocks, 2 * L.bwp, L.bwp, w.xbc, w.ld_xbc, L.bwp, w.aux, w.ld_aux, 2 * L.bwp, b.n, s));
  return bb_hy_rglru(&c, &L, &w, &b, s);
}

int mlstm(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  int first = 0, rows = b.n_pre;         // sequences left to the scan; rows whose outputs are still to be normed and gated
  if (b.n_pre > 0 && !c.dtype && L.np <= 128 && L.pp <= 128) {
    BB_TRY(bb_hy_mlstm_gates(&c, &L, &w, b.n_pre, s));
    BB_TRY(bb_mlstm_chunk(&c, &L, &w, &b, s));
    first = b.ns_pre;
    rows = 0;
  }
  const int rc = bb_hy_mlstm_decode(&c, &L, &w, &b, s);
  if (rc == BB_ESIZE) rows = b.n;
  else if (rc) return rc;
  BB_TRY(bb_hy_mlstm_scan(&c, &L, &w, &b, first, (rc == BB_ESIZE ? b.ns : b.ns_pre) - first, s));
  return bb_hy_head_post(&c, &L, &w, rows, s);
}

int gated_linear(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  if (b.n_pre > 0) {
    BB_TRY(project_f32(c, L.w2, at(c, w.proj, L.off_w1), w.ld_proj, w.f32, w.ld_f32, b.n_pre, 1.f, 0, s));
    const int rc = bb_gla_chunk(&c, &L, &w, &b, s);
    if (rc && rc != BB_ESIZE) return rc;
    BB_TRY(bb_hy_linear_scan(&c, &L, &w, &b, rc == BB_OK, s));    // what is left: marked pairs, or fp32 and other sizes
  }
  return bb_hy_linear_decode(&c, &L, &w, &b, s);
}

int retention(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  if (b.n_pre > 0) {
    BB_TRY(bb_hy_turn(&c, &L, &w, &b, s));
    const int rc = bb_retention_chunk(&c, &L, &w, &b, s);
    if (rc == BB_ESIZE) BB_TRY(bb_hy_linear_scan(&c, &L, &w, &b, 0, s));   // fp32, or sizes the tiles do not cover
    else if (rc) return rc;
    else BB_TRY(bb_hy_linear_post(&c, &L, &w, b.n_pre, s));
  }
  return bb_hy_linear_decode(&c, &L, &w, &b, s);
}

int mixer(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  switch (L.kind) {
    case 0: return attention(c, L, w, b, s);
    case 1: return mamba2(c, L, w, b, s);
    case 2: return latent_attention(c, L, w, b, s);
    case 3: return general_delta(c, L, w, b, s);
    case 4: return rglru(c, L, w, b, s);
    case 5: return mlstm(c, L, w, b, s);
    case 6: return gated_linear(c, L, w, b, s);
    case 7: return retention(c, L, w, b, s);
    default: return BB_EARG;
  }
}

// Small steps leave most of the machine idle, so a layer's feed-forward half runs beside its mixer: on a stream
// of its own, forked behind the norms and joined before the output GEMM (a captured graph gets both branches).
constexpr int BESIDE_ROWS = 256;

struct SideStream {
  cudaStream_t s = nullptr;
  cudaEvent_t fork = nullptr, join = nullptr, ready = nullptr;
};
SideStream* side_stream() {
  static SideStream per_device[64];
  static std::mutex lock;
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return nullptr;
  std::lock_guard<std::mutex> g(lock);
  SideStream& d = per_device[dev];
  if (!d.s && (cudaEventCreateWithFlags(&d.fork, cudaEventDisableTiming) != cudaSuccess ||
               cudaEventCreateWithFlags(&d.join, cudaEventDisableTiming) != cudaSuccess ||
               cudaEventCreateWithFlags(&d.ready, cudaEventDisableTiming) != cudaSuccess ||
               cudaStreamCreateWithFlags(&d.s, cudaStreamNonBlocking) != cudaSuccess))
    return nullptr;
  return &d;
}
#define BB_CUDA(expr)                           \
  do {                                          \
    const cudaError_t e_ = (expr);              \
    if (e_ != cudaSuccess) return (int)e_;      \
  } while (0)

int feed_forward(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  BB_TRY(project(c, L.up, w.h2, c.dp, at(c, w.proj, L.off_up), w.ld_proj, b.n, s));
  return bb_hy_polynorm(&c, &L, &w, b.n, s);
}

int forward_depth(const BbHyCfg& c, const BbHyWork& w, const BbHyBatch& b, float* trace, void* s) {
  const size_t level = (size_t)w.rows * c.dp;
  SideStream* side = b.n <= BESIDE_ROWS ? side_stream() : nullptr;
  for (int li = 0; li < c.n_layers; ++li) {
    const BbHyLayer& L = c.layers[li];
    BB_TRY(bb_hy_mix_norm(&c, li, &w, &b, trace && li ? trace + (size_t)(li - 1) * b.n * c.dp : nullptr, s));
    const bool fork = side && L.ff > 0;
    if (fork) {
      BB_CUDA(cudaEventRecord(side->fork, (cudaStream_t)s));
      BB_CUDA(cudaStreamWaitEvent(side->s, side->fork, 0));
      BB_TRY(feed_forward(c, L, w, b, side->s));
      BB_CUDA(cudaEventRecord(side->join, side->s));
    }
    BB_TRY(project(c, L.in, w.h, c.dp, w.proj, w.ld_proj, b.n, s));
    BB_TRY(mixer(c, L, w, b, s));
    if (fork) BB_CUDA(cudaStreamWaitEvent((cudaStream_t)s, side->join, 0));
    else if (L.ff > 0) BB_TRY(feed_forward(c, L, w, b, s));
    BB_TRY(project_f32(c, L.out, w.cat, w.ld_cat, w.x + (li + 1) * level, c.dp, b.n, 1.f, 1, s));
  }
  if (trace) {
    BbHyBatch all = b;      // the last layer's sum for every row
    all.want = nullptr;
    all.n_want = b.n < w.want_rows ? b.n : w.want_rows;
    BB_TRY(bb_hy_mix_norm(&c, c.n_layers, &w, &all, trace + (size_t)(c.n_layers - 1) * b.n * c.dp, s));
  }
  return bb_hy_mix_norm(&c, c.n_layers, &w, &b, nullptr, s);
}

// y = x W_g^T per 128-row tile of the experts' rows
int project_tiles(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const void* weights, int n, int k, const void* x, int ldx,
                  void* y, int ldy, int tiles, void* s) {
  if (c.dtype)
    return bb_sgemm_tiles(static_cast<const float*>(x), static_cast<const float*>(weights), static_cast<float*>(y), tiles * 128, n, k,
                          ldx, ldy, w.ex_tile, s);
  // tile width: enough tiles to fill the machine
  const int sms = sm_count();
  const int bn = n >= 256 && tiles * ((n + 255) / 256) >= sms ? 256 : (n >= 128 && tiles * ((n + 127) / 128) >= sms / 2 ? 128 : 64);
  return bb_gemm_bf16_grouped(x, weights, y, tiles * 128, n, k, ldx, k, ldy, 0, 0, 1, w.ex_tile, n, L.n_experts * n, nullptr, 0, 0, bn,
                              s);
}

constexpr int ROUTE_ROWS = 128;    // rows up to which these products run as slices of channels

// fp32 products of the normed input, and every token's experts
int route(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  const int rc = b.n <= ROUTE_ROWS ? bb_hy_route_row(&c, &L, &w, b.n, s) : BB_ESIZE;
  if (rc != BB_ESIZE) return rc;
  BB_TRY(project_f32(c, L.in32, w.h, c.dp, w.f32, w.ld_f32, b.n, 1.f, 0, s));
  return L.n_experts > 0 ? bb_hy_route(&c, &L, &w, b.n, s) : BB_OK;
}

// Every token's experts -> their outputs in w.ex_out, and the rows there
int experts(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, void* s) {
  const int tiles = bb_hy_moe_tiles(&L, b.n);
  BB_TRY(bb_hy_expert_rows(&c, &L, &w, b.n, s));
  BB_TRY(project_tiles(c, L, w, L.w_egu, 2 * L.effp, c.dp, w.ex_in, c.dp, w.ex_gu, w.ld_gu, tiles, s));
  BB_TRY(bb_hy_expert_glu(&c, &L, &w, b.n, s));
  return project_tiles(c, L, w, L.w_edown, c.dp, L.effp, w.ex_act, w.ld_act, w.ex_out, c.dp, tiles, s);
}

// Layers that hy_start begins.  In small steps the fp32 products and the experts run beside the mixer.
int forward_start(const BbHyCfg& c, const BbHyWork& w, const BbHyBatch& b, float* trace, void* s) {
  SideStream* side = b.n <= BESIDE_ROWS ? side_stream() : nullptr;
  const cudaStream_t main = (cudaStream_t)s;
  const size_t level = (size_t)b.n * c.dp;
  if (trace && b.n_want < b.n) return BB_EARG;       // the last layer's trace goes through the wanted rows' buffer
  for (int li = 0; li < c.n_layers; ++li) {
    const BbHyLayer& L = c.layers[li];
    BB_TRY(bb_hy_start(&c, li, &w, &b, 0, trace && li ? trace + (li - 1) * level : nullptr, s));
    const bool fork = side && L.n_experts > 0;
    void* t = s;
    if (fork) {
      t = side->s;
      BB_CUDA(cudaEventRecord(side->fork, main));
      BB_CUDA(cudaStreamWaitEvent(side->s, side->fork, 0));
    }
    if (L.in32.w) BB_TRY(route(c, L, w, b, t));
    const bool gates = L.kind == 5 || (L.beside && L.beside->kind == 5);
    if (fork && gates) BB_CUDA(cudaEventRecord(side->ready, side->s));
    if (L.n_experts > 0) BB_TRY(experts(c, L, w, b, t));
    if (fork) BB_CUDA(cudaEventRecord(side->join, side->s));
    BB_TRY(project(c, L.in, w.h, c.dp, w.proj, w.ld_proj, b.n, s));
    if (fork && gates) BB_CUDA(cudaStreamWaitEvent(main, side->ready, 0));
    BB_TRY(mixer(c, L, w, b, s));
    if (L.beside) {
      BbHyWork v = w;
      v.cat = at(c, w.cat, L.beside->off_cat);
      BB_TRY(mixer(c, *L.beside, v, b, s));
    }
    if (L.kind != 0 && L.ff > 0) BB_TRY(bb_hy_glu(&c, &L, &w, b.n, s));
    BB_TRY(project_f32(c, L.out, w.cat, w.ld_cat, w.x, c.dp, b.n, c.residual_mult, 1, s));
    if (fork) BB_CUDA(cudaStreamWaitEvent(main, side->join, 0));
  }
  if (trace) BB_TRY(bb_hy_start(&c, c.n_layers, &w, &b, 1, trace + (c.n_layers - 1) * level, s));
  return bb_hy_start(&c, c.n_layers, &w, &b, 0, nullptr, s);
}

// A sublayer's result: y = x W^T, or in small steps added into zeros.
int project_y(const BbHyCfg& c, const BbHyLin& L, const void* x, int ldx, void* y, float* y32, int rows, void* s) {
  return hy_sums_y(c, rows) ? project_f32(c, L, x, ldx, y32, c.dp, rows, 1.f, 1, s) : project(c, L, x, ldx, y, c.dp, rows, s);
}

// gelu(x W^T)
int project_gelu(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, int rows, void* s) {
  if (!c.dtype)
    return bb_gemm_bf16(w.h, L.up.w, w.cat, nullptr, rows, L.up.n, L.up.k, c.dp, L.up.k, w.ld_cat, 0, 0, 3, 1.f, 0, 0, s);
  BB_TRY(project(c, L.up, w.h, c.dp, w.proj, w.ld_proj, rows, s));
  return bb_hy_gelu(&c, &L, &w, rows, s);
}

// Layers with several residual streams: mixer, then feed-forward, hy_streams before each and behind the last.  In small
// steps mixers side by side run on two streams of the device.
int forward_streams(const BbHyCfg& c, const BbHyWork& w, const BbHyBatch& b, float* trace, void* s) {
  SideStream* side = b.n <= BESIDE_ROWS ? side_stream() : nullptr;
  const cudaStream_t main = (cudaStream_t)s;
  const size_t level = (size_t)b.n * c.dp;
  const BbHyLayer* before = nullptr;
  int fq = 0;
  for (int li = 0; li < c.n_layers; ++li) {
    const BbHyLayer& L = c.layers[li];
    BB_TRY(bb_hy_streams(&c, before, fq, &L, 0, &w, &b, 0, trace && li ? trace + (li - 1) * level : nullptr, s));
    BB_TRY(bb_hy_shift(&c, &L, &w, &b, s));
    BB_TRY(project(c, L.in, w.h, c.dp, w.proj, w.ld_proj, b.n, s));
    if (L.beside) {
      BbHyWork v = w;
      v.cat = at(c, w.cat, L.beside->off_cat);
      const cudaStream_t t = side ? side->s : main;
      if (side) {
        BB_CUDA(cudaEventRecord(side->fork, main));
        BB_CUDA(cudaStreamWaitEvent(side->s, side->fork, 0));
      }
      BB_TRY(mixer(c, *L.beside, v, b, t));
      BB_TRY(project_y(c, L.beside->out, v.cat, w.ld_cat, w.yb, w.yb32, b.n, t));
      if (side) BB_CUDA(cudaEventRecord(side->join, side->s));
    }
    BB_TRY(mixer(c, L, w, b, s));
    BB_TRY(project_y(c, L.out, w.cat, w.ld_cat, w.ya, w.ya32, b.n, s));
    if (L.beside && side) BB_CUDA(cudaStreamWaitEvent(main, side->join, 0));
    before = &L;
    fq = 0;
    if (L.n_experts > 0 || L.down.w) {
      BB_TRY(bb_hy_streams(&c, before, fq, &L, 1, &w, &b, 0, nullptr, s));
      fq = 1;
      if (L.n_experts > 0) {
        BB_TRY(route(c, L, w, b, s));
        BB_TRY(experts(c, L, w, b, s));
      } else {
        BB_TRY(project_gelu(c, L, w, b.n, s));
        BB_TRY(project_y(c, L.down, w.cat, w.ld_cat, w.ya, w.ya32, b.n, s));
      }
    }
  }
  if (trace) BB_TRY(bb_hy_streams(&c, before, fq, nullptr, 0, &w, &b, 1, trace + (c.n_layers - 1) * level, s));
  return bb_hy_streams(&c, before, fq, nullptr, 0, &w, &b, 0, nullptr, s);
}

}  // namespace

// One step.  Logits land in w->logits [n_want, vocabp]; `trace` (may be null): fp32 [n_layers][n][dp]
// copies of the residual stream after every layer.
BB_API int bb_hybrid_forward(const BbHyCfg* c, const BbHyWork* w, const BbHyBatch* b, float* trace, void* stream) {
  if (!c || !w || !b || b->n <= 0 || b->n > w->rows || b->n_want > w->want_rows) return BB_EARG;
  if (c->streams > 0 || c->depth_avg || !c->embed_norm) {
    BB_TRY(c->streams > 0 ? forward_streams(*c, *w, *b, trace, stream)
                          : (c->depth_avg ? forward_depth : forward_start)(*c, *w, *b, trace, stream));
    if (b->n_want <= 0) return BB_OK;
    const BbHyLin head{c->head, c->vocabp, c->dp};
    BB_TRY(project_f32(*c, head, w->hn, c->dp, w->logits, c->vocabp, b->n_want, 1.f, 0, stream));
    return bb_hy_cap(c, w, b->n_want, stream);
  }
  BB_TRY(bb_hy_embed_norm(c, b->tok, w->x, b->n, stream));
  for (int li = 0; li < c->n_layers; ++li) {
    const BbHyLayer& L = c->layers[li];
    BB_TRY(bb_hy_norm(c->dtype, w->x, nullptr, L.norm, w->h, b->n, c->width, c->dp, c->eps, stream));
    BB_TRY(project(*c, L.in, w->h, c->dp, w->proj, w->ld_proj, b->n, stream));
    BB_TRY(mixer(*c, L, *w, *b, stream));
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
  out[4] = sizeof(BbPooled);
  return BB_OK;
}

// Structures of the hybrid decoder's native forward (recurrent and attention layers with a parallel
// feed-forward), shared by the layer sequence and its kernels and mirrored field for field by the
// ctypes classes in brain_b200/serve/hybrid_native.py.
//
// Every matrix is stored with both extents padded to multiples of 8 (zero rows / columns), so the
// sections of a fused projection start on 16-byte boundaries and padded columns are zero throughout.
// dtype 0: bf16 activations, weights and K/V pages; dtype 1: fp32 throughout.
#pragma once
#include <cstddef>
#include <cstdint>

struct BbHyLin {
  const void* w;   // [n, k]
  int n, k;
};

struct BbHyLayer {
  int kind;            // 0 attention, 1 mamba2, 2 latent attention, 3 generalised delta rule, 4 gated linear recurrence,
                       // 5 matrix memory (mLSTM), 6 gated linear attention, 7 retention
  const float* norm;   // [dp] gain of the layer's norm (one already added where it is stored around 0)
  BbHyLin in;          // every projection that reads the normed input, stacked along the rows
  BbHyLin out;         // mixer output projection | feed-forward down projection, side by side
  // feed-forward (ff = 0: none): columns of its halves in the projection and of its product in `cat`
  int ff, off_gate, off_up, off_act;
  float glu_limit, glu_alpha, glu_shift;
  // attention
  int hq, hk, dk, dv, dkp, dvp;            // true and padded head sizes
  int off_q, off_k, off_v, off_g;          // columns of the projection
  const float *q_norm, *k_norm;            // [hq dkp] / [hk dkp] gains of the whole-projection norm
  const float *cos_t, *sin_t;              // [max_pos][rot / 2]
  int rot;                                 // rotated leading dimensions of a head (0: none)
  float scale, softcap;                    // softcap <= 0: none
  float vmix;
  int v_role;                              // 0 plain, 1 stores its values for later layers, 2 mixes them in
  void *kc, *vc;                           // pages [blocks][hk][block_size][dkp | dvp]
  // mamba2
  int heads, p, n, groups, taps, norm_groups;
  int inner, innerp, ch, chp;              // heads * p, padded; convolved channels, padded
  int off_z, off_xbc, off_dt;
  const float *conv_w, *conv_b;            // [taps][chp], [chp]
  const float *dt_bias, *a, *d_skip;       // [heads]; a = -exp(A_log)
  const float* gnorm;                      // [innerp]
  void* conv_state;                        // [slots][max(taps - 1, 1)][chp]: raw inputs, position p at p % (taps - 1)
  float* ssm_state;                        // [slots][heads][n][p]; 3: [slots][heads][p][p]; 4: [slots][chp]
  // a feed-forward with a norm and a GEMM of its own: polynomial of root-mean-square norms
  const float* norm2;                      // [dp] (null: the feed-forward reads the mixer's norm)
  BbHyLin up;                              // [ffp, dp]; its output takes columns off_up of the projection
  const float *up_b, *down_b;              // [ffp], [dp]; down_b is added where the layer's residual starts
  const float* poly;                       // [4]
  // depth average: weights of the results so far, [layer index + 2]
  const float* dwa;
  // latent attention (hq heads; dk / dkp unrotated, rot / rotp rotated, dv / dvp value sizes; one page row
  // per token in kc: latent | rotated key part, kvrp + rotp wide)
  int qr, qrp, kvr, kvrp, rotp, own_kv, window;   // window 0: every earlier key
  int off_dq, off_ckv;
  const float *dq_norm, *dkv_norm;         // [qrp], [kvrp]
  BbHyLin uq;                              // [hq (dkp + rotp), qrp]
  const void *w_abs;                       // [hq][kvrp][dkp]: queries into the latents' space
  const void *w_uv;                        // [hq][dvp][kvrp]: values out of it
  BbHyLin expand;                          // [hq (dkp + rotp) | hq dvp, kvrp + rotp]: keys and values of page rows
  // generalised delta rule (heads of p, padded pp)
  int pp, wr, wrp;                         // ... and the rank of its decay
  int off_r, off_kk, off_vv, off_gg, off_a, off_w1;
  BbHyLin w2;                              // [heads pp, wrp]
  const float *w0, *a_b;                   // [heads pp]
  // gated linear recurrence (blocks of bw channels, padded bwp; chp = innerp = blocks bwp)
  int blocks, bw, bwp, off_y;
  const float *y_b, *x_b;                  // [chp]
  const void* w_gate;                      // [blocks][2 bwp][bwp]: recurrence gate rows, then input gate rows
  const float *r_b, *i_b, *lam;            // [chp]; lam = decay constant times softplus of the parameter
  // a second mixer that reads the same input; its output takes the columns of `cat` from its off_cat on
  const BbHyLayer* beside;
  int off_cat;
  // attention: sigmoid gate at off_g (0 none, 1 one value per head, 2 one per element of the output), a factor
  // on the output, biases [hq dkp] / [hk dkp] / [hk dvp] (null: none; q_norm and k_norm null: no norms)
  int gate_kind;
  float out_scale;
  const float *q_b, *k_b, *v_b;
  // feed-forward: 0 clamped gated unit, 1 gelu(gate) up; biases [ffp] (null: none; up_b as above)
  int glu_kind;
  const float* gate_b;
  // products of the normed input that stay fp32: router logits, then the raw gates of a matrix memory
  BbHyLin in32;
  int off32_i, off32_f;
  // matrix memory (heads of n query / key channels, padded np, and p value channels, padded pp): keys at
  // off_kk, queries right behind them at off_q, values off_vv, output gate off_gg; i_b and f_b [heads].
  // State [slots][heads][mem >= n p + n + 1, a multiple of 4]: matrix, normaliser, running maximum
  int np, mem;
  float gate_cap, q_scale;
  const float* f_b;
  // mixture of experts (n_experts = 0: none): [experts][gate effp | up effp][dp], [experts][dp][effp]
  int n_experts, top, groups_all, groups_keep, eff, effp;
  float route_scale, route_tiny, e_limit, e_alpha, e_shift;
  const void *w_egu, *w_edown;
  // scores of a router: 0 softmax, over the sum of the chosen ones; 1 the sigmoid of each.  weigh_input: a row's weight
  // multiplies what its expert reads (the outputs are then summed as they are)
  int score_kind, weigh_input;
  // residual streams: biases of the norms [dp], token shift [dp] (null: none) and the last input before it
  // [slots][dp], connections of the mixer and the feed-forward: [in s | out s | mix s s, from and to]
  const float *norm_b, *norm2_b, *shift;
  void* shift_state;
  const float *hc[2];
  BbHyLin down;                            // of a feed-forward that follows its mixer (its `up` above)
  const float* out_gain;                   // [dp] mixers side by side, each result normed (null: as it is)
  // attention: norms per head (q_norm [dkp], k_norm [dkp] for every head), neighbouring pairs rotated; the means of
  // blocks of `pool` tokens in pages of pool_rows rows, each in the page of its last token; a number per head [hq] in
  // the softmax's denominator; tables [max_pos][dv / 2] that turn values, and outputs back (null: none)
  int head_norm, pool, pool_rows;
  void *pkc, *pvc;                         // [blocks][hk][pool_rows][dkp | dvp]
  const float *sink, *vcos_t, *vsin_t;
  // linear attention (heads of n key channels, padded np, and p value channels, padded pp; columns and state as a
  // matrix memory's, the state without normaliser): decays sigmoid(z)^decay_root with z = w2 (columns off_w1) + w0, or
  // constants: keep_less [heads] = decay - 1, a = its logarithm; gate silu(columns off_gg), gnorm [heads pp] or null
  float decay_root;
  const float* keep_less;
};

struct BbHyCfg {
  int dtype, width, dp, vocab, vocabp, n_layers, block_size;
  float eps, residual_mult;
  const void* embed;                       // [vocab, dp]
  const float *embed_norm, *final_norm;    // [dp]
  const void* head;                        // [vocabp, dp]
  const BbHyLayer* layers;
  const void* pos;                         // [max positions, dp] added to the embedding (null: none)
  int max_pos;
  float embed_scale;
  int depth_avg;                           // layers pass on weighted sums of all results (see BbHyWork::x)
  int streams;                             // copies of the residual stream (0: one, without connections)
  const float* final_norm_b;               // [dp] (null: none)
  float logit_cap;                         // logits become cap tanh(logits / cap) (0: as they are)
};

// One packed batch: rows of prompt portions first (n_pre rows of ns_pre sequences), then one row for
// every decoding sequence.
struct BbHyBatch {
  const int *tok, *pos, *row_seq;          // [n]
  const int *seq_row0;                     // [ns + 1]
  const int *seq_pos0, *seq_ctx, *seq_slot;  // [ns] first position, context after the step, state slot
  const int* tables;                       // [ns, max_blocks]
  const int *tile_seq, *tile_qt;           // 128-row query tiles of the prompt portions
  const int *want;                         // [n_want] rows whose logits are asked for (null: every row)
  // page rows whose keys and values prompt portions multiply out: n_exp rows of the page pool, of sequence
  // s from kv_row0[s], the first of them at position kv_pos0[s]
  const int *exp_src, *kv_row0, *kv_pos0;
  int n_exp;
  int max_blocks, n, n_pre, ns, ns_pre, n_tiles, n_want, max_len;   // max_len: longest portion
  const int* ctx_row0;                     // [ns_pre] sum of the contexts of the portions before
  int max_ctx;                             // longest context of a portion
};

struct BbHyWork {
  float* x;          // [rows, dp] residual stream; with depth averages [n_layers + 1][rows, dp]: the
                     // embedding, then every layer's result; with several streams [rows][streams][dp]
  void* h;           // [rows, dp]
  void* proj;        // [rows, ld_proj]
  void* cat;         // [rows, ld_cat]
  void* xbc;         // [rows, ld_xbc]
  float* dt;         // [rows, ld_dt]
  void* y;           // [rows, ld_y]
  void* v_first;     // [rows, ld_v]
  float *part_o, *part_ml;   // decode attention partials
  float* seg;        // chunked state-space scratch
  long seg_floats;
  void* hn;          // [want, dp]
  float* logits;     // [want, vocabp]
  int rows, want_rows, ld_proj, ld_cat, ld_xbc, ld_dt, ld_y, ld_v, splits;
  int pool_blocks;
  // second normed input, latent attention (queries, absorbed queries, latent outputs; gathered page rows and
  // their keys and values), and gate / decay projections of the recurrences
  void *h2, *q, *qa, *ol, *ckv, *kvx, *aux;
  int ld_q, ld_qa, ld_ol, ld_ckv, ld_kvx, ld_aux, exp_rows;
  // fp32 products of the normed input; mixture of experts: rows sorted by expert, every expert's on 128-row
  // tiles of their own (input, both halves, their product, output), and of every (token, choice) its expert, row
  // and weight; rows of every expert; expert of every tile (-1: unused), then how many rows every tile has
  float *f32, *part32;                     // [rows, ld_f32]; slices of the same for few rows
  long part32_floats;
  void *ex_in, *ex_gu, *ex_act, *ex_out;   // [moe_rows, dp | ld_gu | ld_act | dp]
  int *pair_expert, *pair_row;             // [rows top]
  float* pair_w;
  int *ex_count, *ex_tile;                 // [experts], [2][moe_rows / 128]
  int ld_f32, ld_gu, ld_act, moe_rows;
  // residual streams: results of a sublayer [rows, dp] (two of mixers side by side), in small bf16 steps (hy_sums_y) added
  // up in fp32 where hy_streams has left zeros; pooled keys and values that prompt
  // portions see, [pk_rows, ld_pk], of sequence s from ctx_row0[s] / pool on
  void *ya, *yb, *pk;
  float *ya32, *yb32;
  int ld_pk, pk_rows;
  // chunks of gated linear attention: [n_pre / 128 + ns_pre][heads][n][p] and marks [..][heads]
  float* chunks;
  int* chunk_flags;
  long chunk_floats, chunk_marks;
};

// Steps of few rows whose projections into the streams are cut along their inner extent, to fill the machine.
static inline bool hy_sums_y(const BbHyCfg& c, int rows) { return !c.dtype && rows <= 256; }

// Rows and pitch of a latent attention layer's queries: through their own latent, or straight from the input.
static inline void* hy_latent_queries(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, int* ld) {
  *ld = L.uq.w ? w.ld_q : w.ld_proj;
  return L.uq.w ? w.q : static_cast<char*>(w.proj) + (size_t)L.off_q * (c.dtype ? 4 : 2);
}

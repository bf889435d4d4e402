// What attention over a window may have beside it: means of blocks of tokens behind the window, a sink in the
// softmax's denominator, rotated values.  Mirrored by brain_b200/serve/hybrid_native.py.
#pragma once

struct BbPooled {
  int pool, pool_rows;       // blocks of `pool` tokens (0: none); the means of a block lie in the page of its last token
  const void *pkc, *pvc;     // ([blocks][kv heads][pool_rows][head size]), at that token's offset / pool
  const void* pk;            // prompts: the means that queries see as rows [pk_rows, ld_pk], keys | values of all heads,
  int ld_pk, pk_rows;        // those of sequence s from pool_row0[s] / pool on
  const int* pool_row0;
  const float* sink;         // [query heads] (null: none)
  const float *vcos, *vsin;  // tables [position][vturn / 2] that turn outputs back by their row's angles (null: none)
  int vturn;
};

"""ctypes mirrors of ``csrc/serve/hybrid.hpp`` and the packing of a hybrid decoder's weights into what the
native forward reads: per layer ONE matrix of everything that reads the normed input and ONE of what is
added to the residual stream, all extents padded to multiples of 8 with zeros."""
from __future__ import annotations

import ctypes as C
from typing import List, Tuple

import torch

P, I, F = C.c_void_p, C.c_int, C.c_float


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class Lin(C.Structure):
    _fields_ = [("w", P), ("n", I), ("k", I)]


class Layer(C.Structure):
    _fields_ = [("kind", I), ("norm", P), ("inp", Lin), ("out", Lin),
                ("ff", I), ("off_gate", I), ("off_up", I), ("off_act", I),
                ("glu_limit", F), ("glu_alpha", F), ("glu_shift", F),
                ("hq", I), ("hk", I), ("dk", I), ("dv", I), ("dkp", I), ("dvp", I),
                ("off_q", I), ("off_k", I), ("off_v", I), ("off_g", I),
                ("q_norm", P), ("k_norm", P), ("cos_t", P), ("sin_t", P), ("rot", I),
                ("scale", F), ("softcap", F), ("vmix", F), ("v_role", I), ("kc", P), ("vc", P),
                ("heads", I), ("p", I), ("n", I), ("groups", I), ("taps", I), ("norm_groups", I),
                ("inner", I), ("innerp", I), ("ch", I), ("chp", I),
                ("off_z", I), ("off_xbc", I), ("off_dt", I),
                ("conv_w", P), ("conv_b", P), ("dt_bias", P), ("a", P), ("d_skip", P), ("gnorm", P),
                ("conv_state", P), ("ssm_state", P),
                ("norm2", P), ("up", Lin), ("up_b", P), ("down_b", P), ("poly", P), ("dwa", P),
                ("qr", I), ("qrp", I), ("kvr", I), ("kvrp", I), ("rotp", I), ("own_kv", I), ("window", I),
                ("off_dq", I), ("off_ckv", I), ("dq_norm", P), ("dkv_norm", P), ("uq", Lin), ("w_abs", P), ("w_uv", P),
                ("expand", Lin), ("pp", I), ("wr", I), ("wrp", I),
                ("off_r", I), ("off_kk", I), ("off_vv", I), ("off_gg", I), ("off_a", I), ("off_w1", I),
                ("w2", Lin), ("w0", P), ("a_b", P),
                ("blocks", I), ("bw", I), ("bwp", I), ("off_y", I), ("y_b", P), ("x_b", P), ("w_gate", P),
                ("r_b", P), ("i_b", P), ("lam", P),
                ("beside", P), ("off_cat", I), ("gate_kind", I), ("out_scale", F), ("q_b", P), ("k_b", P), ("v_b", P),
                ("glu_kind", I), ("gate_b", P), ("in32", Lin), ("off32_i", I), ("off32_f", I),
                ("np", I), ("mem", I), ("gate_cap", F), ("q_scale", F), ("f_b", P),
                ("n_experts", I), ("top", I), ("groups_all", I), ("groups_keep", I), ("eff", I), ("effp", I),
                ("route_scale", F), ("route_tiny", F), ("e_limit", F), ("e_alpha", F), ("e_shift", F),
                ("w_egu", P), ("w_edown", P), ("score_kind", I), ("weigh_input", I),
                ("norm_b", P), ("norm2_b", P), ("shift", P), ("shift_state", P), ("hc", P * 2), ("down", Lin), ("out_gain", P),
                ("head_norm", I), ("pool", I), ("pool_rows", I), ("pkc", P), ("pvc", P), ("sink", P), ("vcos_t", P), ("vsin_t", P),
                ("decay_root", F), ("keep_less", P)]


#: pages and slots of a layer
CACHES = ("kc", "vc", "pkc", "pvc", "conv_state", "ssm_state", "shift_state")


class Cfg(C.Structure):
    _fields_ = [("dtype", I), ("width", I), ("dp", I), ("vocab", I), ("vocabp", I), ("n_layers", I),
                ("block_size", I), ("eps", F), ("residual_mult", F), ("embed", P), ("embed_norm", P),
                ("final_norm", P), ("head", P), ("layers", P), ("pos", P), ("max_pos", I), ("embed_scale", F), ("depth_avg", I),
                ("streams", I), ("final_norm_b", P), ("logit_cap", F)]


class Batch(C.Structure):
    _fields_ = [(n, P) for n in ("tok", "pos", "row_seq", "seq_row0", "seq_pos0", "seq_ctx", "seq_slot", "tables",
                                 "tile_seq", "tile_qt", "want", "exp_src", "kv_row0", "kv_pos0")] + \
               [(n, I) for n in ("n_exp", "max_blocks", "n", "n_pre", "ns", "ns_pre", "n_tiles", "n_want", "max_len")] + \
               [("ctx_row0", P), ("max_ctx", I)]


class Work(C.Structure):
    _fields_ = [(n, P) for n in ("x", "h", "proj", "cat", "xbc", "dt", "y", "v_first", "part_o", "part_ml", "seg")] + \
               [("seg_floats", C.c_long), ("hn", P), ("logits", P)] + \
               [(n, I) for n in ("rows", "want_rows", "ld_proj", "ld_cat", "ld_xbc", "ld_dt", "ld_y", "ld_v", "splits",
                                 "pool_blocks")] + \
               [(n, P) for n in ("h2", "q", "qa", "ol", "ckv", "kvx", "aux")] + \
               [(n, I) for n in ("ld_q", "ld_qa", "ld_ol", "ld_ckv", "ld_kvx", "ld_aux", "exp_rows")] + \
               [("f32", P), ("part32", P), ("part32_floats", C.c_long)] + \
               [(n, P) for n in ("ex_in", "ex_gu", "ex_act", "ex_out", "pair_expert", "pair_row", "pair_w", "ex_count",
                                 "ex_tile")] + \
               [(n, I) for n in ("ld_f32", "ld_gu", "ld_act", "moe_rows")] + \
               [("ya", P), ("yb", P), ("pk", P), ("ya32", P), ("yb32", P), ("ld_pk", I), ("pk_rows", I),
                ("chunks", P), ("chunk_flags", P), ("chunk_floats", C.c_long), ("chunk_marks", C.c_long)]


class Pooled(C.Structure):
    """``csrc/common/pooled.hpp``: what attention over a window has beside it."""
    _fields_ = [("pool", I), ("pool_rows", I), ("pkc", P), ("pvc", P), ("pk", P), ("ld_pk", I), ("pk_rows", I), ("pool_row0", P),
                ("sink", P), ("vcos", P), ("vsin", P), ("vturn", I)]


def padded_rows(w: torch.Tensor, heads: int, size: int, sizep: int) -> torch.Tensor:
    """[heads * size, k] -> [heads * sizep, k], zero rows after every head."""
    if size == sizep:
        return w
    out = w.new_zeros(heads, sizep, w.shape[1])
    out[:, :size] = w.view(heads, size, w.shape[1])
    return out.view(heads * sizep, w.shape[1])


def padded_groups(w: torch.Tensor, rows_p: int, cols_p: int) -> torch.Tensor:
    """[groups, rows, cols] -> [groups, rows_p, cols_p], zeros around every matrix."""
    g, r, c = w.shape
    if (r, c) == (rows_p, cols_p):
        return w.contiguous()
    out = w.new_zeros(g, rows_p, cols_p)
    out[:, :r, :c] = w
    return out


class RowStack:
    """Row sections of one fused matrix, each starting at a multiple of 8."""

    def __init__(self):
        self.parts: List[torch.Tensor] = []
        self.n = 0

    def add(self, w: torch.Tensor) -> int:
        off = self.n
        r = pad8(w.shape[0])
        if r != w.shape[0]:
            w = torch.cat([w, w.new_zeros(r - w.shape[0], w.shape[1])])
        self.parts.append(w)
        self.n += r
        return off

    def matrix(self, kp: int) -> torch.Tensor:
        w = torch.cat(self.parts)
        if w.shape[1] != kp:
            w = torch.cat([w, w.new_zeros(w.shape[0], kp - w.shape[1])], dim=1)
        return w.contiguous()


def vec(t: torch.Tensor, n: int, dev) -> torch.Tensor:
    """fp32 vector on the device, zero-padded to ``n``."""
    out = torch.zeros(n, dtype=torch.float32)
    out[:t.numel()] = t.detach().float().reshape(-1).cpu()
    return out.to(dev)


def head_vec(t: torch.Tensor, heads: int, size: int, sizep: int, dev) -> torch.Tensor:
    """fp32 [heads * sizep] gains from [heads * size], zero in the padding."""
    return padded_rows(t.detach().float().reshape(-1, 1), heads, size, sizep).reshape(-1).contiguous().to(dev)


def columns(sections: List[Tuple[torch.Tensor, int]], np_: int) -> torch.Tensor:
    """[np_, sum of widths] matrix of column sections (matrix, padded width)."""
    total = sum(w for _, w in sections)
    first = sections[0][0]
    out = first.new_zeros(np_, total)
    o = 0
    for m, w in sections:
        out[:m.shape[0], o:o + m.shape[1]] = m
        o += w
    return out.contiguous()


def check_layout(lib) -> None:
    """The mirrors above have the library's structure sizes (a stale build raises here, not on the GPU)."""
    out = (C.c_int * 5)()
    lib.bb_hybrid_sizes(out)
    mine = [C.sizeof(s) for s in (Layer, Cfg, Batch, Work, Pooled)]
    if list(out) != mine:
        raise RuntimeError(f"hybrid structures: library {list(out)}, binding {mine}; rebuild the native library")

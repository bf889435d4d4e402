"""Serving engine of the hybrid decoders (Pakalix, Nezalorn, Zepesun, Povipel): pages for the attention layers, recurrent-state
slots for the recurrent layers, one native call per step.

* A step is ONE packed batch: prompt portions of any length and single decoded tokens of several
  sequences run together (``csrc/serve/hybrid_forward.cu``).  Every entry point - the scheduler's prefill,
  mixed and decode calls and :meth:`HybridEngine.step_logits` - goes through it.
* Pages: per attention layer keys and values ``[num_blocks + 1, kv_heads, block_size, head size]``, per latent
  attention layer with latents of its own ``[num_blocks + 1, block_size, latent | rotated key part]``; where blocks of
  tokens are pooled behind a window, their means ``[num_blocks + 1, kv_heads, ceil(block_size / pool), head size]``,
  each in the page of the block's last token, so that the tokens' page table names them.
  State slots: per recurrent layer the fp32 state (``[heads, state, head size]``, ``[heads, key, value]``, a
  matrix memory with its normaliser and running maximum, or one value per channel) and, where it has a
  convolution, a ring of the last taps - 1 raw inputs; with a token shift the last input of every layer.  A sequence
  at position 0 starts from zeros, so pages and slots are reused as they are.
* Layers that run several times share their weights; every pass is a layer of its own here, with its own pages and
  slots.
* Mixtures of experts: rows of a step sorted by expert onto 128-row tiles, one grouped product per matrix.
* ``dtype='bf16'``: bf16 weights, activations, pages and convolution inputs; the residual stream, norms,
  rotation, scores, softmax, routers, step sizes, gates of a recurrence, decays and the recurrent state are
  fp32.  ``dtype='fp32'``: everything in fp32, no tensor-core rounding."""
from __future__ import annotations

import ctypes as C
import time
from typing import Dict, List, NamedTuple, Optional, Sequence

import numpy as np
import torch

from ..models.config import HybridConfig
from ..ops import _cuda
from ..ops import functional as F
from ..ops._cuda import NativeError, stream_ptr
from . import hybrid_native as hn
from .base import PagedEngineBase
from .hybrid_native import pad8

_MAX_SPLITS = 16


class Entry(NamedTuple):
    """The next tokens of one sequence in a step."""
    tokens: np.ndarray
    start: int                   # position of the first of them
    block_table: np.ndarray
    slot: int
    want: Sequence[int]          # places among them whose logits are asked for


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


class _Scratch:
    """Device buffers of a step of up to ``rows`` rows, ``want`` logit rows, ``dec`` decode rows and ``exp``
    page rows whose keys and values are multiplied out."""

    def __init__(self, eng: "HybridEngine", rows: int, want: int, dec: int, exp: int, portions: bool = True):
        dev, dt = eng.device, eng.dtype
        m = eng.ld
        self.rows, self.want, self.dec, self.exp = rows, want, dec, exp
        z = lambda *s, dtype=dt: torch.zeros(*s, device=dev, dtype=dtype)
        f32 = torch.float32
        traits = eng.cfg.traits
        self.x = z(eng.cfg.n_layers + 1 if traits.depth_average else eng.cfg.streams, rows, eng.dp, dtype=f32)
        self.h, self.h2 = z(rows, eng.dp), z(rows if traits.two_norms or traits.token_shift and portions else 1, eng.dp)
        self.ya, self.yb = (z(rows if traits.streams else 1, eng.dp) for _ in range(2))
        self.ya32, self.yb32 = (z(min(rows, 256) if traits.streams else 1, eng.dp, dtype=f32) for _ in range(2))
        self.pk = z(max(exp, 1) if portions else 1, m["pk"])
        self.proj, self.cat = z(rows, m["proj"]), z(rows, m["cat"])
        self.xbc, self.dt, self.y = z(rows, m["xbc"]), z(rows, m["dt"], dtype=f32), z(rows, m["y"])
        self.v_first = z(rows, m["v"])
        # latent attention: absorbed queries are needed for decoded rows only where portions multiply keys out
        ab = rows if eng.absorb_portions else max(dec, 1)
        self.q, self.qa, self.ol, self.aux = z(rows, m["q"]), z(ab, m["qa"]), z(ab, m["ol"]), z(rows, m["aux"])
        self.ckv, self.kvx = z(max(exp, 1), m["ckv"]), z(max(exp, 1), m["kvx"])
        self.f32 = z(rows, m["f32"], dtype=f32)
        self.part32 = z(max(-(-eng.dp // 64) * min(rows, 128) * max(l.in32.n for l in eng.layers), 1), dtype=f32)
        # mixture of experts: every expert that has rows takes at most one 128-row tile that is not full
        routed = [l for l in eng.layers if l.n_experts]
        top = max((l.top for l in routed), default=0)
        moe = 128 * max((rows * l.top // 128 + min(rows * l.top, l.n_experts) for l in routed), default=0)
        i32 = torch.int32
        self.ex_in, self.ex_out = (z(max(moe, 1), eng.dp if routed else 8) for _ in range(2))
        self.ex_gu, self.ex_act = z(max(moe, 1), m["gu"]), z(max(moe, 1), m["act"])
        self.pair_expert, self.pair_row = (z(max(rows * top, 1), dtype=i32) for _ in range(2))
        self.pair_w = z(max(rows * top, 1), dtype=f32)
        self.ex_count = z(max((l.n_experts for l in routed), default=1), dtype=i32)
        self.ex_tile = z(max(moe // 64, 1), dtype=i32)
        po = pm = 1
        for l in eng.mixers:
            if l.kind == 0 and dec and not eng.fp32:
                n = dec * l.hq * self._max_splits(l.hk, dec)
                po, pm = max(po, n * (64 if l.dvp <= 64 else 128)), max(pm, n * 2)
            if l.kind == 2 and dec and not eng.fp32:
                n = dec * l.hq * _MAX_SPLITS
                po, pm = max(po, n * l.kvrp), max(pm, n * 2)
        self.part_o, self.part_ml = z(po, dtype=f32), z(pm, dtype=f32)
        # segment states of the chunked recurrence (prompt portions): two machine-fulls of states
        npmax = max([l.mem if l.kind == 5 else l.n * l.p for l in eng.mixers if l.kind in (1, 5, 7) and max(l.n, l.p) <= 128],
                    default=0)
        self.seg = z(2 * 2 * eng.sm_count * (npmax + 1) if portions and not eng.fp32 and npmax else 1, dtype=f32)
        # chunks of gated linear attention, one sequence's last ones not full
        gla = [l for l in eng.mixers if l.kind == 6 and l.np <= 64 and l.pp <= 128] if portions and not eng.fp32 else []
        slots = rows // 128 + 32
        self.chunks = z(max((slots * l.heads * l.n * l.p for l in gla), default=1), dtype=f32)
        self.chunk_flags = z(max((slots * l.heads for l in gla), default=1), dtype=i32)
        self.hn, self.logits = z(max(want, 1), eng.dp), z(max(want, 1), eng.vocabp, dtype=f32)
        w = self.work = hn.Work()
        for n in ("x", "h", "proj", "cat", "xbc", "dt", "y", "v_first", "part_o", "part_ml", "seg", "hn", "logits", "h2", "q",
                  "qa", "ol", "aux", "ckv", "kvx", "f32", "part32", "ex_in", "ex_gu", "ex_act", "ex_out", "pair_expert", "pair_row",
                  "pair_w", "ex_count", "ex_tile", "ya", "yb", "ya32", "yb32", "pk", "chunks",
                  "chunk_flags"):
            setattr(w, n, _ptr(getattr(self, n)))
        w.chunk_floats, w.chunk_marks = self.chunks.numel(), self.chunk_flags.numel()
        w.seg_floats, w.part32_floats = self.seg.numel(), self.part32.numel()
        w.rows, w.want_rows, w.exp_rows, w.moe_rows, w.pk_rows = rows, max(want, 1), exp, moe, self.pk.shape[0]
        for k in m:
            setattr(w, "ld_" + k, m[k])
        w.splits, w.pool_blocks = _MAX_SPLITS, eng.num_blocks + 1

    @staticmethod
    def _max_splits(hk: int, dec: int) -> int:
        """The most K/V splits a batch of up to ``dec`` rows takes, as rows * splits is what counts."""
        return max(1, -(-min(_MAX_SPLITS * dec, 4 * 160 // hk + dec + 1) // dec))


class HybridEngine(PagedEngineBase):
    def __init__(self, model, block_size: int = 16, num_blocks: int = 1024, max_seq_len: int = 4096,
                 max_prefill: int = 512, weights: str = "bf16", topk: int = 64, tp=None, cuda_graphs: bool = True,
                 kv_dtype: str = "bf16", kv_clip=None, state_slots: int = 16, dtype: str = "bf16", device=None):
        cfg: HybridConfig = model.cfg
        if weights != "bf16" or kv_dtype != "bf16" or kv_clip is not None:
            raise ValueError("hybrid decoders are served with unquantised weights and K/V pages")
        if tp is not None and tp.world > 1:
            raise ValueError("hybrid decoders are served on one GPU")
        if dtype not in ("bf16", "fp32"):
            raise ValueError(f"dtype {dtype!r}: bf16 or fp32")
        dev = torch.device(device) if device is not None else next(model.parameters()).device
        if dev.type != "cuda":
            raise NativeError("the hybrid engine runs on CUDA devices only (its kernels have no CPU form)")
        self.cfg, self.device, self.cuda = cfg, dev, True
        self.fp32 = dtype == "fp32"
        self.dtype = torch.float32 if self.fp32 else torch.bfloat16
        self.vocab, self.vocabp = cfg.vocab, pad8(cfg.vocab)
        self.dp = pad8(cfg.width)
        self.block_size, self.num_blocks = block_size, num_blocks
        self.max_seq_len, self.max_prefill_tokens = min(max_seq_len, cfg.max_position_embeddings), max_prefill
        max_seq_len = self.max_seq_len
        self.topk_capacity = topk
        self.max_blocks = (max_seq_len + block_size - 1) // block_size
        self.state_slots, self.dummy_slot = state_slots, state_slots
        self.dummy_block = num_blocks      # padded rows of a bucketed decode batch live there
        self.sm_count = torch.cuda.get_device_properties(dev).multi_processor_count
        self._init_common(cuda_graphs)
        self._keep: List[torch.Tensor] = []
        self._scratch: Dict[tuple, _Scratch] = {}
        self._iota: Dict[int, torch.Tensor] = {}
        self._rope: Dict[tuple, tuple] = {}
        self._pack(model)
        hn.check_layout(_cuda.lib())
        self._forward = _cuda.lib().bb_hybrid_forward
        self._forward.restype = C.c_int

    # ------------------------------------------------------------------ weights
    def _hold(self, t: torch.Tensor) -> int:
        self._keep.append(t)
        return t.data_ptr()

    def _hold_matrix(self, t: torch.Tensor) -> int:
        self._matrix_bytes += t.numel() * t.element_size()
        return self._hold(t)

    def _lin(self, w: torch.Tensor) -> hn.Lin:
        return hn.Lin(self._hold_matrix(w), w.shape[0], w.shape[1])

    def _mat(self, name: str) -> torch.Tensor:
        return self._tensor(name).detach().to(self.device, self.dtype)

    def _vec(self, t: torch.Tensor, n: int) -> int:
        return self._hold(hn.vec(t, n, self.device))

    def _head_vec(self, name: str, heads: int, size: int) -> int:
        return self._hold(hn.head_vec(self._tensor(name), heads, size, pad8(size), self.device))

    def _rows(self, name: str, heads: int, size: int) -> torch.Tensor:
        return hn.padded_rows(self._mat(name), heads, size, pad8(size))

    def _cols(self, name: str, heads: int, size: int) -> torch.Tensor:
        """An output projection with its input columns padded head by head."""
        return hn.padded_rows(self._mat(name).t().contiguous(), heads, size, pad8(size)).t()

    def _widest(self, **kw) -> None:
        for k, n in kw.items():
            self.ld[k] = max(self.ld[k], n)

    def _pages(self, *shape) -> int:
        t = torch.zeros(self.num_blocks + 1, *shape, device=self.device, dtype=self.dtype)
        self.kv_bytes += t.numel() * t.element_size()
        self._caches[t.data_ptr()] = lambda: self._pages(*shape)
        return self._hold(t)

    def _slots(self, *shape, dtype=torch.float32) -> int:
        t = torch.zeros(self.state_slots + 1, *shape, device=self.device, dtype=dtype)
        self.state_bytes += t.numel() * t.element_size()
        self._caches[t.data_ptr()] = lambda: self._slots(*shape, dtype=dtype)
        return self._hold(t)

    def _pass(self, dst, src) -> None:
        """``dst``: another pass of layer ``src``, the same weights with pages and slots of its own."""
        C.memmove(C.byref(dst), C.byref(src), C.sizeof(src))
        for name in hn.CACHES:
            p = getattr(src, name)
            if p:
                setattr(dst, name, self._caches[p]())
        if src.beside:
            side = hn.Layer()
            self._pass(side, hn.Layer.from_address(src.beside))
            self.mixers.append(side)
            dst.beside = C.addressof(side)

    def _angles(self, rot):
        key = (rot.dims, rot.base, str(rot.scaling))
        if key not in self._rope:
            f, mag = rot.frequencies()
            ang = torch.arange(self.max_blocks * self.block_size, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
            self._rope[key] = tuple((mag * t).float().to(self.device) for t in (ang.cos(), ang.sin()))
        return map(_ptr, self._rope[key])

    def _rotary(self, L, rot) -> None:
        L.cos_t, L.sin_t, L.rot = *self._angles(rot), rot.dims

    def _paired_rows(self, w: torch.Tensor, heads: int, rot) -> torch.Tensor:
        """Rows of a projection in the order in which a rotated pair's are neighbours."""
        if rot is None or rot.interleaved:
            return w
        per = w.view(heads, -1, w.shape[1])
        half = rot.dims // 2
        order = [i // 2 + (i % 2) * half for i in range(rot.dims)] + list(range(rot.dims, per.shape[1]))
        return per[:, order].reshape(w.shape)

    # Every packer adds what reads the normed input to ``stack`` (to ``stack32`` where the product stays fp32) and
    # returns the mixer's output projection with its padded input width.  ``scale``: a factor on the mixer's result.
    def _pack_attention(self, i: int, L, m, p: str, stack, scale: float = 1.0):
        dkp, dvp = pad8(m.dim), pad8(m.vdim)
        L.kind, L.hq, L.hk, L.dk, L.dv, L.dkp, L.dvp = 0, m.heads, m.kv_heads, m.dim, m.vdim, dkp, dvp
        L.off_q = stack.add(self._rows(p + "q", m.heads, m.dim))
        L.off_k = stack.add(self._rows(p + "k", m.kv_heads, m.dim))
        L.off_v = stack.add(self._rows(p + "v", m.kv_heads, m.vdim))
        elems = m.gate == "element"
        if m.gate is not None:
            L.off_g = stack.add(self._rows(p + "g", m.heads, m.vdim) if elems else self._mat(p + "g"))
        L.gate_kind, L.out_scale, L.window = (2 if elems else 1) if m.gate is not None else 0, scale, m.window or 0
        if m.qk_norm == "head":
            L.head_norm, L.q_norm, L.k_norm = 1, *(self._vec(self._tensor(p + n + ".norm"), dkp) for n in "qk")
            if m.rot is not None and not m.rot.interleaved:
                raise ValueError("attention with norms per head rotates neighbouring pairs")
        elif m.qk_norm:
            L.q_norm, L.k_norm = self._head_vec(p + "q.norm", m.heads, m.dim), self._head_vec(p + "k.norm", m.kv_heads, m.dim)
        if m.bias:
            L.q_b, L.k_b, L.v_b = (self._head_vec(p + n + ".b", h, d) for n, h, d in
                                   (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim), ("v", m.kv_heads, m.vdim)))
            self.out_bias.append(scale * self._tensor(p + "o.b").float().cpu())
        if m.rot is not None and m.rot.dims:
            self._rotary(L, m.rot)
        L.scale, L.softcap = m.scale, m.softcap or 0.0
        first = next((j for j, l in enumerate(self.cfg.layers) if l.mixer.kind == "attention" and l.mixer.v_mix), None)
        L.v_role = 0 if not m.v_mix else (1 if i == first else 2)
        L.vmix = float(self._tensor(p + "vmix").float()) if m.v_mix else 0.0
        L.kc, L.vc = (self._pages(m.kv_heads, self.block_size, d) for d in (dkp, dvp))
        if m.pool is not None:
            L.pool, L.pool_rows = m.pool, -(-self.block_size // m.pool)
            L.pkc, L.pvc = (self._pages(m.kv_heads, L.pool_rows, d) for d in (dkp, dvp))
            self.least_pool = min(self.least_pool or m.pool, m.pool)
            self._widest(pk=m.kv_heads * (dkp + dvp))
        if m.sink:
            L.sink = self._vec(self._tensor(p + "sink"), m.heads)
        if m.value_rot is not None:
            L.vcos_t, L.vsin_t = self._angles(m.value_rot)
        self._widest(v=m.kv_heads * dvp)
        return self._cols(p + "o", m.heads, m.vdim), m.heads * dvp

    def _pack_mamba2(self, i: int, L, m, p: str, stack):
        inner, ch = m.inner, m.channels
        L.kind, L.heads, L.p, L.n, L.groups = 1, m.heads, m.vdim, m.state, m.groups
        L.taps, L.norm_groups = m.conv, m.norm_groups
        L.inner, L.innerp, L.ch, L.chp = inner, pad8(inner), ch, pad8(ch)
        w_in = self._mat(p + "in")
        L.off_z = stack.add(w_in[:inner])
        L.off_xbc = stack.add(w_in[inner:inner + ch])
        L.off_dt = stack.add(w_in[inner + ch:])
        T = self._tensor
        self._pack_conv(L, T(p + "conv"), T(p + "conv.b"), 1, ch)
        L.dt_bias = self._vec(T(p + "dt_bias"), pad8(m.heads))
        L.a = self._vec(-torch.exp(T(p + "A_log").detach().double()).float(), pad8(m.heads))
        L.d_skip = self._vec(T(p + "D"), pad8(m.heads))
        L.gnorm = self._vec(T(p + "norm"), pad8(inner))
        L.ssm_state = self._slots(m.heads, m.state, m.vdim)
        self._widest(dt=pad8(m.heads), y=pad8(inner))
        return self._mat(p + "o"), pad8(inner)

    def _pack_conv(self, L, w: torch.Tensor, b: torch.Tensor, blocks: int, size: int) -> None:
        """Short convolution over ``blocks`` x ``size`` channels, padded block by block."""
        taps, chp = w.shape[1], blocks * pad8(size)
        cw = hn.padded_rows(w.detach().float().cpu(), blocks, size, pad8(size)).t()
        L.conv_w = self._hold(cw.contiguous().to(self.device))
        L.conv_b = self._hold(hn.head_vec(b, blocks, size, pad8(size), self.device))
        L.conv_state = self._slots(max(taps - 1, 1), chp, dtype=self.dtype)
        self._widest(xbc=chp)

    def _pack_latent_attention(self, i: int, L, m, p: str, stack):
        H, dkp, rotp, dvp, kvrp, qrp = m.heads, *map(pad8, (m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank if m.q_latent else 0))
        L.kind, L.hq, L.hk, L.dk, L.dkp, L.dv, L.dvp = 2, H, 1, m.dim, dkp, m.vdim, dvp
        L.out_scale = 1.0
        L.qr, L.qrp, L.kvr, L.kvrp, L.rotp, L.scale, L.window = m.q_rank, qrp, m.kv_rank, kvrp, rotp, m.scale, m.window or 0
        self._rotary(L, m.rot)
        # the kernels rotate neighbouring pairs: half-split ones are brought there by the order of the rows
        R = m.rot_dim
        order = list(range(R)) if m.rot.interleaved else [i // 2 + (i % 2) * (R // 2) for i in range(R)]
        per_head = lambda name, n: self._mat(p + name).view(H, n, -1)
        q = per_head("uq" if m.q_latent else "q", m.dim + R)
        qin = qrp if m.q_latent else q.shape[2]
        q = torch.cat([hn.padded_groups(q[:, :m.dim], dkp, qin), hn.padded_groups(q[:, m.dim:][:, order], rotp, qin)],
                      dim=1).view(-1, qin)
        if m.q_latent:
            L.off_dq = stack.add(self._mat(p + "dq"))
            L.dq_norm = self._vec(self._tensor(p + "dq.norm"), qrp)
            L.uq = self._lin(q)
            self._widest(q=H * (dkp + rotp))
        else:
            L.off_q = stack.add(q)
        if m.head_gate:
            L.gate_kind, L.off_g = 1, stack.add(self._mat(p + "g"))
        row = kvrp + rotp
        if m.kv_from is None:
            w = self._mat(p + "dkv")
            L.own_kv, L.off_ckv = 1, stack.add(w[:m.kv_rank])
            stack.add(w[m.kv_rank:][order])
            L.dkv_norm = self._vec(self._tensor(p + "dkv.norm"), kvrp)
            L.kc = self._pages(self.block_size, row)
        else:
            L.kc = self.layers[m.kv_from].kc
        uk, uv = per_head("uk", m.dim), per_head("uv", m.vdim)
        L.w_abs = self._hold_matrix(hn.padded_groups(uk.transpose(1, 2), kvrp, dkp))
        L.w_uv = self._hold_matrix(hn.padded_groups(uv, dvp, kvrp))
        fits = not self.fp32 and dkp + rotp <= 128 and dvp <= 128       # sizes of the tensor-core prefill
        if fits:
            # one matrix makes keys and values of page rows; the rotated part passes through its identity
            k = uk.new_zeros(H, dkp + rotp, row)
            k[:, :m.dim, :m.kv_rank] = uk
            k[:, dkp:dkp + m.rot_dim, kvrp:kvrp + m.rot_dim] = torch.eye(m.rot_dim, device=k.device, dtype=k.dtype)
            v = hn.padded_groups(uv, dvp, row)
            L.expand = self._lin(torch.cat([k.view(-1, row), v.view(-1, row)]).contiguous())
            self._widest(ckv=row, kvx=H * (dkp + rotp + dvp))
        self._widest(qa=H * row, ol=H * kvrp)
        self.absorb_portions |= not fits
        self.exp_window = None if m.window is None or self.exp_window is None else max(self.exp_window, m.window)
        return self._cols(p + "o", H, m.vdim), H * dvp

    def _pack_general_delta(self, i: int, L, m, p: str, stack):
        pp = pad8(m.dim)
        L.kind, L.heads, L.p, L.pp, L.inner, L.innerp = 3, m.heads, m.dim, pp, m.inner, m.heads * pp
        L.off_r, L.off_kk, L.off_vv, L.off_gg, L.off_a = (stack.add(self._rows(p + n, m.heads, m.dim)) for n in "rkvga")
        L.wr, L.wrp, L.off_w1 = m.decay_rank, pad8(m.decay_rank), stack.add(self._mat(p + "w1"))
        L.w2 = self._lin(hn.columns([(self._rows(p + "w2", m.heads, m.dim), L.wrp)], L.innerp))
        L.w0, L.a_b, L.gnorm = (self._head_vec(p + n, m.heads, m.dim) for n in ("w0", "a.b", "norm"))
        L.ssm_state = self._slots(m.heads, m.dim, m.dim)
        self._widest(aux=L.innerp, y=L.innerp)
        return self._cols(p + "o", m.heads, m.dim), L.innerp

    def _pack_rglru(self, i: int, L, m, p: str, stack):
        B, n = m.blocks, m.width // m.blocks
        np_ = pad8(n)
        L.kind, L.blocks, L.bw, L.bwp, L.taps = 4, B, n, np_, m.conv
        L.inner, L.innerp, L.ch, L.chp = m.width, B * np_, m.width, B * np_
        L.off_y, L.off_xbc = stack.add(self._rows(p + "y", B, n)), stack.add(self._rows(p + "x", B, n))
        L.y_b, L.x_b, L.r_b, L.i_b = (self._head_vec(p + k, B, n) for k in ("y.b", "x.b", "ra.b", "ri.b"))
        self._pack_conv(L, self._tensor(p + "conv"), self._tensor(p + "conv.b"), B, n)
        lam = m.decay * torch.nn.functional.softplus(self._tensor(p + "lam").detach().double())
        L.lam = self._hold(hn.head_vec(lam, B, n, np_, self.device))
        L.w_gate = self._hold_matrix(torch.cat([hn.padded_groups(self._mat(p + k), np_, np_) for k in ("ra", "ri")], dim=1))
        L.ssm_state = self._slots(L.chp)
        self._widest(aux=2 * L.chp)
        return self._cols(p + "o", B, n), L.innerp

    def _pack_mlstm(self, i: int, L, m, p: str, stack, scale: float = 1.0):
        H, np_, pp = m.heads, pad8(m.dim), pad8(m.vdim)
        L.kind, L.heads, L.n, L.np, L.p, L.pp, L.inner, L.innerp = 5, H, m.dim, np_, m.vdim, pp, m.inner, H * pp
        L.groups, L.gate_cap, L.q_scale = H, m.gate_cap, m.dim ** -0.5
        L.off_kk, L.off_q = (stack.add(self._rows(p + n, H, m.dim)) for n in "kq")
        L.off_vv, L.off_gg = (stack.add(self._rows(p + n, H, m.vdim)) for n in "vg")
        L.off32_i, L.off32_f = (self.stack32.add(self._mat(p + n)) for n in "if")
        L.i_b, L.f_b = (self._vec(self._tensor(p + n + ".b"), pad8(H)) for n in "if")
        L.gnorm = self._hold(hn.head_vec(scale * self._tensor(p + "norm").float(), H, m.vdim, pp, self.device))
        L.mem = -(-(m.dim * m.vdim + m.dim + 1) // 4) * 4
        L.ssm_state = self._slots(H, L.mem)
        self._widest(y=L.innerp)
        return self._cols(p + "o", H, m.vdim), L.innerp

    def _pack_linear(self, L, m, p: str, stack, rot=None):
        """What the forms of linear attention have in common: head sizes, projections, state."""
        H, np_, pp = m.heads, pad8(m.dim), pad8(m.vdim)
        L.heads, L.n, L.np, L.p, L.pp, L.inner, L.innerp, L.groups = H, m.dim, np_, m.vdim, pp, m.inner, H * pp, H
        L.q_scale = m.dim ** -0.5
        L.off_kk, L.off_q = (stack.add(hn.padded_rows(self._paired_rows(self._mat(p + n), H, rot), H, m.dim, np_)) for n in "kq")
        L.off_vv, L.off_gg = (stack.add(self._rows(p + n, H, m.vdim)) for n in "vg")
        L.ssm_state = self._slots(H, m.dim, m.vdim)
        self._widest(y=L.innerp)
        return self._cols(p + "o", H, m.vdim), L.innerp

    def _pack_gated_linear(self, i: int, L, m, p: str, stack, scale: float = 1.0):
        out = self._pack_linear(L, m, p, stack)
        H, np_ = m.heads, pad8(m.dim)
        L.kind, L.decay_root = 6, 1.0 / m.tau
        L.wr, L.wrp, L.off_w1 = m.decay_rank, pad8(m.decay_rank), stack.add(self._mat(p + "a1"))
        L.w2 = self._lin(hn.columns([(self._rows(p + "a2", H, m.dim), L.wrp)], H * np_))
        L.w0 = self._head_vec(p + "a2.b", H, m.dim)
        L.gnorm = self._hold(hn.head_vec(scale * self._tensor(p + "norm").float().repeat(H), H, m.vdim, L.pp, self.device))
        self._widest(f32=2 * H * np_)          # z, and in chunks the sums of the decays' logarithms
        return out

    def _pack_retention(self, i: int, L, m, p: str, stack):
        out = self._pack_linear(L, m, p, stack, m.rot)
        decay = torch.tensor(m.decay, dtype=torch.float64)
        L.kind, L.keep_less, L.a = 7, self._vec((decay - 1.0).float(), m.heads), self._vec(decay.log().float(), m.heads)
        if m.rot is not None and m.rot.dims:
            self._rotary(L, m.rot)
        return out

    def _pack_parallel(self, i: int, L, m, p: str, stack):
        ls, rs = (1.0, 1.0) if m.normed else (m.left_scale, m.right_scale)
        left = self._pack_attention(i, L, m.left, p + "left.", stack, ls)
        R = hn.Layer()
        right = getattr(self, "_pack_" + m.right.kind)(i, R, m.right, p + "right.", stack, rs)
        R.off_cat = left[1]
        self.mixers.append(R)                  # (kept alive there)
        L.beside = C.addressof(R)
        if m.normed:                           # each has an output projection of its own, and a gain
            R.out = self._lin(hn.columns([right], self.dp))
            for side, name, s in ((L, "left.out", m.left_scale), (R, "right.out", m.right_scale)):
                side.out_gain = self._vec(s * self._tensor(p + name).float(), self.dp)
            self._widest(cat=left[1] + right[1])
            return [left]
        return [left, right]

    def _pack_routed(self, L, f, p: str) -> None:
        effp, dp, E = pad8(f.expert.ff), self.dp, f.experts
        L.n_experts, L.top, L.groups_all, L.groups_keep, L.eff, L.effp = E, f.top, f.groups, f.keep, f.expert.ff, effp
        L.route_scale, L.route_tiny, L.score_kind, L.weigh_input = f.scale, f.tiny, int(f.scores == "sigmoid"), int(f.weigh_input)
        L.e_limit, L.e_alpha, L.e_shift = f.expert.limit, f.expert.alpha, f.expert.shift
        gu = torch.zeros(E, 2, effp, dp, device=self.device, dtype=self.dtype)
        down = torch.zeros(E, dp, effp, device=self.device, dtype=self.dtype)
        for e in range(E):
            gate, up, out = (self._mat(f"{p}e{e}.{n}") for n in ("gate", "up", "down"))
            gu[e, 0, :f.expert.ff, :gate.shape[1]], gu[e, 1, :f.expert.ff, :up.shape[1]] = gate, up
            down[e, :out.shape[0], :f.expert.ff] = out
        L.w_egu, L.w_edown = self._hold_matrix(gu), self._hold_matrix(down)
        self._widest(gu=2 * effp, act=effp)

    def _pack(self, model) -> None:
        cfg, dev, dp = self.cfg, self.device, self.dp
        traits = cfg.traits
        T = self._tensor = model.tensor
        runs = cfg.runs
        n = len(runs)
        self.layers = (hn.Layer * n)()
        self.layer_list = [self.layers[i] for i in range(n)]
        self._caches = {}                      # of a device pointer: how to make another like it
        self.least_pool = None                 # smallest blocks that a layer pools
        self.mixers = list(self.layer_list)    # and the second mixers of layers that have two
        self.ld = dict.fromkeys(("proj", "cat", "xbc", "dt", "y", "v", "q", "qa", "ol", "ckv", "kvx", "aux", "f32", "gu", "act", "pk"), 8)
        self.kv_bytes = self.state_bytes = self._matrix_bytes = 0
        # prompt portions of latent attention: whether they also take the absorbed form, and how many keys the
        # widest window of a layer holds (None: all)
        self.absorb_portions, self.exp_window = False, 1
        gain = lambda name: self._vec(traits.norm_offset + T(name).float(), dp)
        bias = lambda name: self._vec(T(name + ".b"), dp) if traits.layer_norm else None
        for run, i in enumerate(runs):
            first = runs.index(i)
            if first < run:
                self._pass(self.layers[run], self.layers[first])
                continue
            L, p, spec = self.layers[run], f"l{i}.", cfg.layers[i]
            L.norm, L.norm_b = gain(p + "norm1"), bias(p + "norm1")
            if traits.token_shift:
                L.shift, L.shift_state = self._vec(T(p + "shift"), dp), self._slots(dp, dtype=self.dtype)
            stack, self.stack32, self.out_bias = hn.RowStack(), hn.RowStack(), []
            f, fp = spec.mlp, p + "mlp."
            if f is not None and f.kind == "routed":
                self.stack32.add(self._mat(fp + "router"))
                self._pack_routed(L, f, fp)
                f, fp = f.shared, fp + "shared."
            sections = getattr(self, "_pack_" + spec.mixer.kind)(i, L, spec.mixer, p + "mix.", stack)
            sections = sections if isinstance(sections, list) else [sections]
            width = stack.n
            if traits.streams:                 # a feed-forward behind the mixer, each spread over the streams
                for q in range(2 if spec.mlp is not None else 1):
                    L.hc[q] = self._hold(torch.cat([T(f"{p}hc{q + 1}.{k}").float().reshape(-1) for k in ("in", "out", "mix")]).to(dev))
                if spec.mlp is not None:
                    L.norm2, L.norm2_b = gain(p + "norm2"), bias(p + "norm2")
                if f is not None:
                    ffp = pad8(f.ff)
                    L.up = self._lin(hn.columns([(self._mat(fp + "up"), dp)], ffp))
                    L.down = self._lin(hn.columns([(self._mat(fp + "down"), ffp)], dp))
                    self._widest(proj=ffp, cat=ffp)
            elif f is not None:
                ffp = pad8(f.ff)
                L.ff, L.off_act = f.ff, sum(w for _, w in sections)
                if f.kind == "polynorm":
                    L.norm2 = gain(p + "norm2")
                    L.up = self._lin(hn.columns([(self._mat(fp + "up"), dp)], ffp))
                    L.up_b = self._vec(T(fp + "up.b"), ffp)
                    L.poly, L.off_up = self._vec(T(fp + "act"), 4), stack.n
                    width = stack.n + ffp
                else:
                    if f.kind == "clamped_glu":
                        L.glu_limit, L.glu_alpha, L.glu_shift = f.limit, f.alpha, f.shift
                    else:
                        L.glu_kind, L.gate_b, L.up_b = 1, self._vec(T(fp + "gate.b"), ffp), self._vec(T(fp + "up.b"), ffp)
                    L.off_gate, L.off_up = stack.add(self._mat(fp + "gate")), stack.add(self._mat(fp + "up"))
                    width = stack.n
                if f.kind != "clamped_glu":
                    self.out_bias.append(T(fp + "down.b").float().cpu())
                sections.append((self._mat(fp + "down"), ffp))
            if self.out_bias:
                L.down_b = self._vec(sum(self.out_bias), dp)
            if traits.depth_average:
                L.dwa = self._vec(T(p + "dwa"), i + 2)
            L.inp, L.out = self._lin(stack.matrix(dp)), self._lin(hn.columns(sections, dp))
            self._widest(proj=width, cat=L.out.k, f32=self.stack32.n)
            if self.stack32.n:
                L.in32 = self._lin(self.stack32.matrix(dp))
        c = self.ccfg = hn.Cfg()
        c.dtype, c.width, c.dp, c.vocab, c.vocabp = int(self.fp32), cfg.width, dp, cfg.vocab, self.vocabp
        c.n_layers, c.block_size, c.eps, c.residual_mult = n, self.block_size, cfg.eps, cfg.residual_mult
        c.depth_avg, c.streams, c.logit_cap = int(traits.depth_average), cfg.streams if traits.streams else 0, cfg.logit_softcap or 0.0
        pad_cols = lambda name: self._hold_matrix(hn.columns([(self._mat(name), dp)], self.vocabp))
        c.embed = pad_cols("embed")
        if traits.positions:
            pos = torch.zeros(cfg.max_position_embeddings, dp, device=dev, dtype=self.dtype)
            pos[:, :cfg.width] = self._mat("pos")
            c.pos, c.max_pos = self._hold_matrix(pos), cfg.max_position_embeddings
        c.embed_scale = cfg.embed_scale
        c.head = c.embed if traits.tied else pad_cols("head")
        c.embed_norm = gain("embed.norm") if traits.embed_norm else None
        c.final_norm, c.final_norm_b = gain("final.norm"), bias("final.norm")
        c.layers = C.cast(self.layers, C.c_void_p)
        del self._tensor, self.stack32, self.out_bias, self._caches

    # ------------------------------------------------------------------ accounting
    def kv_pool_bytes(self) -> int:
        return self.kv_bytes

    def weight_bytes(self) -> int:
        return self._matrix_bytes

    # ------------------------------------------------------------------ steps
    def _scratch_for(self, key, rows: int, want: int, dec: int, exp: int = 0) -> _Scratch:
        s = self._scratch.get(key)
        if s is None or s.rows < rows or s.want < want or s.dec < dec or s.exp < exp:
            if torch.cuda.is_current_stream_capturing():
                raise RuntimeError("step buffers must exist before graph capture")
            if s is not None:
                rows, want, dec, exp = max(rows, s.rows), max(want, s.want), max(dec, s.dec), max(exp, s.exp)
            s = self._scratch[key] = _Scratch(self, rows, want, dec, exp, portions=key == "step")
        return s

    def _run(self, sc: _Scratch, b: hn.Batch, trace: Optional[torch.Tensor] = None) -> torch.Tensor:
        rc = self._forward(C.byref(self.ccfg), C.byref(sc.work), C.byref(b), C.c_void_p(_ptr(trace)), stream_ptr())
        _cuda.launch_count += 1
        if rc != 0:
            raise NativeError(f"bb_hybrid_forward failed with code {rc}")
        self.steps += 1
        return sc.logits[:b.n_want, :self.vocab]

    def _step(self, entries: Sequence[Entry], trace: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Run one packed step; fp32 logits [wanted, vocab] on the device in entry order (a view of step
        buffers: valid until the next step)."""
        sc, b, blob = self._prepare(entries)
        out = self._run(sc, b, trace)
        self._last_blob = blob        # stays alive until the step's kernels are behind the next one
        return out

    def _prepare(self, entries: Sequence[Entry]):
        """Check and pack a step: (step buffers, batch structure, the device memory it points into)."""
        # portions first, single tokens after them: the latter take the decode kernels
        order = [i for i, e in enumerate(entries) if len(e.tokens) > 1]
        ns_pre = len(order)
        order += [i for i, e in enumerate(entries) if len(e.tokens) == 1]
        if len(order) != len(entries):
            raise ValueError("an entry of a step needs at least one token")
        lens = [len(entries[i].tokens) for i in order]
        row0 = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
        n, ns = int(row0[-1]), len(order)
        n_pre = int(row0[ns_pre])
        starts = np.array([entries[i].start for i in order], dtype=np.int32)
        ctx = starts + np.array(lens, dtype=np.int32)
        if int(ctx.max()) > self.max_seq_len:
            raise ValueError(f"{int(ctx.max())} tokens exceed the engine's context of {self.max_seq_len}")
        tok = np.concatenate([np.asarray(entries[i].tokens, dtype=np.int32) for i in order])
        if int(tok.min()) < 0 or int(tok.max()) >= self.vocab:
            raise ValueError("token outside the vocabulary")
        pos = np.concatenate([np.arange(s, s + l, dtype=np.int32) for s, l in zip(starts.tolist(), lens)])
        row_seq = np.repeat(np.arange(ns, dtype=np.int32), lens)
        slot = np.array([entries[i].slot for i in order], dtype=np.int32)
        if ns and (int(slot.min()) < 0 or int(slot.max()) > self.state_slots):
            raise ValueError("state slot out of range")
        tables = np.full((ns, self.max_blocks), -1, dtype=np.int32)
        for r, i in enumerate(order):
            bt = np.asarray(entries[i].block_table, dtype=np.int32)
            used = -(-int(ctx[r]) // self.block_size)
            if used > len(bt) or int(bt[:used].min()) < 0 or int(bt[:used].max()) > self.num_blocks:
                raise ValueError("block table does not cover the step's tokens")
            tables[r, :used] = bt[:used]
        tiles = [(s, q) for s in range(ns_pre) for q in range(-(-lens[s] // 128))]
        # tiles that see the most keys first, so the tail of the launch is short tiles
        tiles.sort(key=lambda t: -(int(starts[t[0]]) + min(lens[t[0]], (t[1] + 1) * 128)))
        first_row = {i: int(row0[r]) for r, i in enumerate(order)}
        want = [first_row[i] + int(w) for i, e in enumerate(entries) for w in e.want]
        exp_src, kv_row0, kv_pos0 = self._expansion(starts[:ns_pre], ctx[:ns_pre], tables)
        parts = [tok, pos, row_seq, row0, starts, ctx, slot, tables.reshape(-1),
                 np.array([t[0] for t in tiles], dtype=np.int32), np.array([t[1] for t in tiles], dtype=np.int32),
                 np.array(want, dtype=np.int32), exp_src, kv_row0, kv_pos0,
                 np.concatenate([[0], np.cumsum(ctx[:ns_pre])]).astype(np.int32)]
        offs = np.concatenate([[0], np.cumsum([-(-p.size // 4) * 4 for p in parts])]).astype(np.int64)
        blob = np.zeros(int(offs[-1]), dtype=np.int32)
        for o, p in zip(offs[:-1].tolist(), parts):
            blob[o:o + p.size] = p
        d_blob = torch.from_numpy(blob).to(self.device)
        base = d_blob.data_ptr()
        b = hn.Batch()
        for name, o in zip(("tok", "pos", "row_seq", "seq_row0", "seq_pos0", "seq_ctx", "seq_slot", "tables", "tile_seq",
                            "tile_qt", "want", "exp_src", "kv_row0", "kv_pos0", "ctx_row0"), offs[:-1].tolist()):
            setattr(b, name, base + 4 * o)
        b.max_blocks, b.n, b.n_pre, b.ns, b.ns_pre = self.max_blocks, n, n_pre, ns, ns_pre
        b.n_tiles, b.n_want, b.max_len, b.n_exp = len(tiles), len(want), max(lens[:ns_pre], default=0), exp_src.size
        b.max_ctx = int(ctx[:ns_pre].max(initial=0))
        pooled = int(ctx[:ns_pre].sum()) // self.least_pool if self.least_pool else 0
        up = lambda v, q: -(-v // q) * q
        sc = self._scratch_for("step", up(n, 256), up(len(want), 16), up(ns - ns_pre, 16) if ns > ns_pre else 0,
                               up(max(exp_src.size, pooled), 256))
        return sc, b, d_blob

    def _expansion(self, starts, ctx, tables):
        """Page rows whose keys and values the prompt portions of latent attention multiply out: for every
        portion its own tokens and the keys that the widest window reaches back to.  Returns (page rows, first
        of them per portion, position of that first)."""
        if self.ld["kvx"] <= 8 or not len(starts):
            return (np.zeros(0, dtype=np.int32),) * 3
        lo = np.zeros_like(starts) if self.exp_window is None else np.maximum(starts - (self.exp_window - 1), 0)
        src = []
        for r, (a, e) in enumerate(zip(lo.tolist(), ctx.tolist())):
            p = np.arange(a, e)
            src.append(tables[r, p // self.block_size] * self.block_size + p % self.block_size)
        row0 = np.concatenate([[0], np.cumsum(ctx - lo)]).astype(np.int32)
        return np.concatenate(src).astype(np.int32), row0, lo.astype(np.int32)

    @torch.no_grad()
    def step_logits(self, entries: Sequence[Entry]) -> torch.Tensor:
        """Feed every entry's tokens in one batch; fp32 logits [wanted, vocab] (device) at the wanted
        places, in the order of the entries and of their ``want`` lists."""
        if self.fault_hook is not None:
            self.fault_hook("prefill")
        return self._step(entries)

    @torch.no_grad()
    def residual_trace(self, tokens: Sequence[int]) -> torch.Tensor:
        """The fp32 residual stream [layer runs, tokens, width] (the sum where there are several) after every layer run
        of one fresh sequence (pages 0.. and the dummy slot are used: for offline inspection of an idle engine)."""
        n = len(tokens)
        out = torch.zeros(len(self.layers), n, self.dp, device=self.device)
        bt = np.arange(self.max_blocks, dtype=np.int32)
        self._step([Entry(np.asarray(tokens, dtype=np.int32), 0, bt, self.dummy_slot, list(range(n)))], out)
        torch.cuda.synchronize()
        return out[:, :, :self.cfg.width]

    # ------------------------------------------------------------------ scheduler's decoder interface
    def _pick(self, logits: torch.Tensor, greedy: bool):
        if greedy:
            return F.argmax_rows(logits), None
        k = min(self.topk_capacity, self.vocab)
        idx, vals = F.topk_rows(logits, k)
        return idx[:, 0].to(torch.int32), (idx, vals)

    def _finish(self, picked, tk):
        toks = picked.cpu().tolist()
        cands = [None] * len(toks)
        if tk is not None:
            idx, vals = tk[0].cpu().tolist(), tk[1].cpu().tolist()
            cands = [list(zip(i, v)) for i, v in zip(idx, vals)]
        return toks, cands

    @torch.no_grad()
    def prefill_chunk(self, tokens: np.ndarray, start: int, block_table: np.ndarray, last: bool, greedy: bool = True,
                      slot: int = 0):
        return self.prefill_batch([(tokens, start, block_table, last, greedy, slot)])[0]

    @torch.no_grad()
    def prefill_batch(self, items):
        """Several prompt portions in one step: items of (tokens, start, block table, last, greedy, state
        slot).  Returns (first token, top-k candidates) per item, (None, None) for portions that do not
        end their prompt."""
        if self.fault_hook is not None:
            self.fault_hook("prefill")
        t0 = time.perf_counter()
        results, _, _ = self._mixed(items, None, None, None, None, all(it[4] for it in items if it[3]))
        a = self.acct
        a["prefill_s"] += time.perf_counter() - t0
        a["prefill_calls"] += 1
        a["prefill_seqs"] += len(items)
        a["prefill_tokens"] += sum(len(it[0]) for it in items)
        return results

    @torch.no_grad()
    def mixed_step(self, items, tokens, positions, block_tables, greedy: bool = True, slots=None):
        """Prompt portions and one decode row per running sequence in one step; arguments and results as
        the dense engine's ``mixed_step``, items with a state slot at the end, ``slots`` of the decode rows."""
        if self.fault_hook is not None:
            self.fault_hook("prefill")
            self.fault_hook("decode")
        t0 = time.perf_counter()
        out = self._mixed(items, tokens, positions, block_tables, slots, greedy)
        a = self.acct
        a["mixed_s"] += time.perf_counter() - t0
        a["mixed_calls"] += 1
        a["prefill_seqs"] += len(items)
        a["prefill_tokens"] += sum(len(it[0]) for it in items)
        a["decode_rows"] += len(tokens)
        return out

    def _mixed(self, items, tokens, positions, block_tables, slots, greedy):
        entries = [Entry(np.asarray(t), int(st), bt, int(slot), [len(t) - 1] if last else [])
                   for t, st, bt, last, _, slot in items]
        nd = 0 if tokens is None else len(tokens)
        for j in range(nd):
            entries.append(Entry(np.asarray(tokens[j:j + 1]), int(positions[j]), block_tables[j], int(slots[j]), [0]))
        logits = self._step(entries)
        final = [i for i, it in enumerate(items) if it[3]]
        results = [(None, None)] * len(items)
        if not final and not nd:
            return results, [], None
        toks, cands = self._finish(*self._pick(logits, greedy))
        for j, i in enumerate(final):
            results[i] = (int(toks[j]), cands[j])
        nf = len(final)
        return results, [[int(t)] for t in toks[nf:]], (None if greedy else cands[nf:])

    def _decode_steps(self, tok, pos, bts, window: int, greedy: bool, slots=None):
        """``window`` decode steps on device tensors -> (tokens [B, window], last top-k or None)."""
        B = tok.shape[0]
        sc = self._scratch_for(("decode", B), B, B, B)
        iota = self._iota.get(B)
        if iota is None:
            iota = self._iota[B] = torch.arange(B + 1, device=self.device, dtype=torch.int32)
        b = hn.Batch()
        b.row_seq, b.seq_row0, b.seq_slot, b.tables = iota.data_ptr(), iota.data_ptr(), slots.data_ptr(), bts.data_ptr()
        b.max_blocks, b.n, b.ns, b.n_want = bts.shape[1], B, B, B
        outs, topks, hold = [], None, []
        for _ in range(window):
            ctx = pos + 1
            hold += [tok, pos, ctx]
            b.tok, b.pos, b.seq_pos0, b.seq_ctx = tok.data_ptr(), pos.data_ptr(), pos.data_ptr(), ctx.data_ptr()
            t, tk = self._pick(self._run(sc, b), greedy)
            outs.append(t)
            topks = tk
            tok, pos = t, ctx
        return torch.stack(outs, dim=1), topks

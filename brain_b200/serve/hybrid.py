"""Serving engine of the hybrid decoders (Pakalix): paged K/V for the attention layers, recurrent-state
slots for the state-space layers, one native call per step.

* A step is ONE packed batch: prompt portions of any length and single decoded tokens of several
  sequences run together (``csrc/serve/hybrid_forward.cu``).  Every entry point - the scheduler's prefill,
  mixed and decode calls and :meth:`HybridEngine.step_logits` - goes through it.
* K/V pages: per attention layer ``[num_blocks + 1, kv_heads, block_size, head size]``.  State slots: per
  state-space layer a ring of the last taps - 1 raw convolution inputs and the fp32 state
  ``[heads, state, head size]``.  A sequence at position 0 starts from zeros, so pages and slots are
  reused as they are.
* ``dtype='bf16'``: bf16 weights, activations, pages and convolution inputs; the residual stream, norms,
  rotation, scores, softmax, step sizes, decays and the recurrent state are fp32.  ``dtype='fp32'``:
  everything in fp32, no tensor-core rounding."""
from __future__ import annotations

import ctypes as C
import time
from typing import Dict, List, NamedTuple, Optional, Sequence

import numpy as np
import torch

from ..models.config import HybridConfig
from ..ops import _cuda
from ..ops import functional as F
from ..ops import reference as ref
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
    """Device buffers of a step of up to ``rows`` rows, ``want`` logit rows and ``dec`` decode rows."""

    def __init__(self, eng: "HybridEngine", rows: int, want: int, dec: int, portions: bool = True):
        dev, dt = eng.device, eng.dtype
        m = eng.ld
        self.rows, self.want, self.dec = rows, want, dec
        z = lambda *s, dtype=dt: torch.zeros(*s, device=dev, dtype=dtype)
        f32 = torch.float32
        self.x, self.h = z(rows, eng.dp, dtype=f32), z(rows, eng.dp)
        self.proj, self.cat = z(rows, m["proj"]), z(rows, m["cat"])
        self.xbc, self.dt, self.y = z(rows, m["xbc"]), z(rows, m["dt"], dtype=f32), z(rows, m["y"])
        self.v_first = z(rows, m["v"])
        po = pm = 1
        for l in eng.layer_list:
            if l.kind == 0 and dec and not eng.fp32:
                n = dec * l.hq * self._max_splits(l.hk, dec)
                po, pm = max(po, n * (64 if l.dvp <= 64 else 128)), max(pm, n * 2)
        self.part_o, self.part_ml = z(po, dtype=f32), z(pm, dtype=f32)
        # segment states of the chunked recurrence (prompt portions): two machine-fulls of states
        npmax = max([l.n * l.p for l in eng.layer_list if l.kind == 1], default=0)
        self.seg = z(2 * 2 * eng.sm_count * (npmax + 1) if portions and not eng.fp32 and npmax <= 128 * 128 else 1, dtype=f32)
        self.hn, self.logits = z(max(want, 1), eng.dp), z(max(want, 1), eng.vocabp, dtype=f32)
        w = self.work = hn.Work()
        for n in ("x", "h", "proj", "cat", "xbc", "dt", "y", "v_first", "part_o", "part_ml", "seg", "hn", "logits"):
            setattr(w, n, _ptr(getattr(self, n)))
        w.seg_floats = self.seg.numel()
        w.rows, w.want_rows = rows, max(want, 1)
        w.ld_proj, w.ld_cat, w.ld_xbc, w.ld_dt, w.ld_y, w.ld_v = (m[k] for k in ("proj", "cat", "xbc", "dt", "y", "v"))
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
        self.max_seq_len, self.max_prefill_tokens = max_seq_len, max_prefill
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

    def _mat(self, t: torch.Tensor) -> torch.Tensor:
        return t.detach().to(self.device, self.dtype)

    def _rope_tables(self, dims: int, base: float):
        key = (dims, base)
        if key not in self._rope:
            self._rope[key] = ref.rope_tables(self.max_seq_len, dims, base, device=self.device)
        return self._rope[key]

    def _pack(self, model) -> None:
        cfg, dev = self.cfg, self.device
        dp, fdt = self.dp, self.dtype
        T = model.tensor
        zeros = lambda *s, dtype=fdt: torch.zeros(*s, device=dev, dtype=dtype)
        n = cfg.n_layers
        self.layers = (hn.Layer * n)()
        self.layer_list = [self.layers[i] for i in range(n)]
        self.ld = dict(proj=8, cat=8, xbc=8, dt=8, y=8, v=8)
        self.kv_bytes = self.state_bytes = 0
        first_values = next((i for i, l in enumerate(cfg.layers) if l.mixer.kind == "attention" and l.mixer.v_mix), None)
        for i, spec in enumerate(cfg.layers):
            L, m, p = self.layers[i], spec.mixer, f"l{i}."
            L.norm = self._hold(hn.vec(1.0 + T(p + "norm1").float(), dp, dev))
            stack = hn.RowStack()
            if m.kind == "attention":
                dkp, dvp = pad8(m.dim), pad8(m.vdim)
                L.kind, L.hq, L.hk, L.dk, L.dv, L.dkp, L.dvp = 0, m.heads, m.kv_heads, m.dim, m.vdim, dkp, dvp
                L.off_q = stack.add(hn.padded_rows(self._mat(T(p + "mix.q")), m.heads, m.dim, dkp))
                L.off_k = stack.add(hn.padded_rows(self._mat(T(p + "mix.k")), m.kv_heads, m.dim, dkp))
                L.off_v = stack.add(hn.padded_rows(self._mat(T(p + "mix.v")), m.kv_heads, m.vdim, dvp))
                L.off_g = stack.add(self._mat(T(p + "mix.g")))
                L.q_norm = self._hold(hn.head_vec(T(p + "mix.q.norm"), m.heads, m.dim, dkp, dev))
                L.k_norm = self._hold(hn.head_vec(T(p + "mix.k.norm"), m.kv_heads, m.dim, dkp, dev))
                if m.rot is not None and m.rot.dims:
                    cos, sin = self._rope_tables(m.rot.dims, m.rot.base)
                    L.cos_t, L.sin_t, L.rot = _ptr(cos), _ptr(sin), m.rot.dims
                L.scale, L.softcap = m.scale, m.softcap or 0.0
                L.v_role = 0 if not m.v_mix else (1 if i == first_values else 2)
                L.vmix = float(T(p + "mix.vmix").float()) if m.v_mix else 0.0
                kc = zeros(self.num_blocks + 1, m.kv_heads, self.block_size, dkp)
                vc = zeros(self.num_blocks + 1, m.kv_heads, self.block_size, dvp)
                L.kc, L.vc = self._hold(kc), self._hold(vc)
                self.kv_bytes += (kc.numel() + vc.numel()) * kc.element_size()
                o = hn.padded_rows(self._mat(T(p + "mix.o")).t().contiguous(), m.heads, m.vdim, dvp).t()
                mixer_w = m.heads * dvp
                self.ld["v"] = max(self.ld["v"], m.kv_heads * dvp)
            else:
                inner, ch = m.inner, m.channels
                L.kind, L.heads, L.p, L.n, L.groups = 1, m.heads, m.vdim, m.state, m.groups
                L.taps, L.norm_groups = m.conv, m.norm_groups
                L.inner, L.innerp, L.ch, L.chp = inner, pad8(inner), ch, pad8(ch)
                w_in = self._mat(T(p + "mix.in"))
                L.off_z = stack.add(w_in[:inner])
                L.off_xbc = stack.add(w_in[inner:inner + ch])
                L.off_dt = stack.add(w_in[inner + ch:])
                cw = torch.zeros(m.conv, pad8(ch))
                cw[:, :ch] = T(p + "mix.conv").detach().float().cpu().t()
                L.conv_w = self._hold(cw.contiguous().to(dev))
                L.conv_b = self._hold(hn.vec(T(p + "mix.conv.b"), pad8(ch), dev))
                L.dt_bias = self._hold(hn.vec(T(p + "mix.dt_bias"), pad8(m.heads), dev))
                L.a = self._hold(hn.vec(-torch.exp(T(p + "mix.A_log").detach().double()).float(), pad8(m.heads), dev))
                L.d_skip = self._hold(hn.vec(T(p + "mix.D"), pad8(m.heads), dev))
                L.gnorm = self._hold(hn.vec(T(p + "mix.norm"), pad8(inner), dev))
                ring = zeros(self.state_slots + 1, max(m.conv - 1, 1), pad8(ch))
                ssm = zeros(self.state_slots + 1, m.heads, m.state, m.vdim, dtype=torch.float32)
                L.conv_state, L.ssm_state = self._hold(ring), self._hold(ssm)
                self.state_bytes += ring.numel() * ring.element_size() + ssm.numel() * 4
                o = self._mat(T(p + "mix.o"))
                mixer_w = pad8(inner)
                self.ld["xbc"] = max(self.ld["xbc"], pad8(ch))
                self.ld["dt"] = max(self.ld["dt"], pad8(m.heads))
                self.ld["y"] = max(self.ld["y"], pad8(inner))
            sections = [(o, mixer_w)]
            if spec.mlp is not None:
                f = spec.mlp
                L.ff, L.glu_limit, L.glu_alpha, L.glu_shift = f.ff, f.limit, f.alpha, f.shift
                L.off_gate = stack.add(self._mat(T(p + "mlp.gate")))
                L.off_up = stack.add(self._mat(T(p + "mlp.up")))
                L.off_act = mixer_w
                sections.append((self._mat(T(p + "mlp.down")), pad8(f.ff)))
            w_in, w_out = stack.matrix(dp), hn.columns(sections, dp)
            L.inp = hn.Lin(self._hold(w_in), w_in.shape[0], w_in.shape[1])
            L.out = hn.Lin(self._hold(w_out), w_out.shape[0], w_out.shape[1])
            self.ld["proj"] = max(self.ld["proj"], w_in.shape[0])
            self.ld["cat"] = max(self.ld["cat"], w_out.shape[1])
        c = self.ccfg = hn.Cfg()
        c.dtype, c.width, c.dp, c.vocab, c.vocabp = int(self.fp32), cfg.width, dp, cfg.vocab, self.vocabp
        c.n_layers, c.block_size, c.eps, c.residual_mult = n, self.block_size, cfg.eps, cfg.residual_mult
        pad_cols = lambda w: hn.columns([(w, dp)], pad8(w.shape[0]))
        c.embed = self._hold(pad_cols(self._mat(T("embed"))))
        c.head = self._hold(pad_cols(self._mat(T("head"))))
        c.embed_norm = self._hold(hn.vec(1.0 + T("embed.norm").float(), dp, dev))
        c.final_norm = self._hold(hn.vec(1.0 + T("final.norm").float(), dp, dev))
        c.layers = C.cast(self.layers, C.c_void_p)

    # ------------------------------------------------------------------ accounting
    def kv_pool_bytes(self) -> int:
        return self.kv_bytes

    def weight_bytes(self) -> int:
        es = 4 if self.fp32 else 2
        n = self.vocabp * self.dp * 2
        for l in self.layer_list:
            n += l.inp.n * l.inp.k + l.out.n * l.out.k
        return n * es

    # ------------------------------------------------------------------ steps
    def _scratch_for(self, key, rows: int, want: int, dec: int) -> _Scratch:
        s = self._scratch.get(key)
        if s is None or s.rows < rows or s.want < want or s.dec < dec:
            if torch.cuda.is_current_stream_capturing():
                raise RuntimeError("step buffers must exist before graph capture")
            if s is not None:
                rows, want, dec = max(rows, s.rows), max(want, s.want), max(dec, s.dec)
            s = self._scratch[key] = _Scratch(self, rows, want, dec, portions=key == "step")
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
        parts = [tok, pos, row_seq, row0, starts, ctx, slot, tables.reshape(-1),
                 np.array([t[0] for t in tiles], dtype=np.int32), np.array([t[1] for t in tiles], dtype=np.int32),
                 np.array(want, dtype=np.int32)]
        offs = np.concatenate([[0], np.cumsum([-(-p.size // 4) * 4 for p in parts])]).astype(np.int64)
        blob = np.zeros(int(offs[-1]), dtype=np.int32)
        for o, p in zip(offs[:-1].tolist(), parts):
            blob[o:o + p.size] = p
        d_blob = torch.from_numpy(blob).to(self.device)
        base = d_blob.data_ptr()
        b = hn.Batch()
        for name, o in zip(("tok", "pos", "row_seq", "seq_row0", "seq_pos0", "seq_ctx", "seq_slot", "tables", "tile_seq",
                            "tile_qt", "want"), offs[:-1].tolist()):
            setattr(b, name, base + 4 * o)
        b.max_blocks, b.n, b.n_pre, b.ns, b.ns_pre = self.max_blocks, n, n_pre, ns, ns_pre
        b.n_tiles, b.n_want, b.max_len = len(tiles), len(want), max(lens[:ns_pre], default=0)
        up = lambda v, q: -(-v // q) * q
        sc = self._scratch_for("step", up(n, 256), up(len(want), 16), up(ns - ns_pre, 16) if ns > ns_pre else 0)
        return sc, b, d_blob

    @torch.no_grad()
    def step_logits(self, entries: Sequence[Entry]) -> torch.Tensor:
        """Feed every entry's tokens in one batch; fp32 logits [wanted, vocab] (device) at the wanted
        places, in the order of the entries and of their ``want`` lists."""
        if self.fault_hook is not None:
            self.fault_hook("prefill")
        return self._step(entries)

    @torch.no_grad()
    def residual_trace(self, tokens: Sequence[int]) -> torch.Tensor:
        """The fp32 residual stream [layers, tokens, width] after every layer of one fresh sequence (pages
        0.. and the dummy slot are used: for offline inspection of an idle engine)."""
        n = len(tokens)
        out = torch.zeros(self.cfg.n_layers, n, self.dp, device=self.device)
        bt = np.arange(self.max_blocks, dtype=np.int32)
        self._step([Entry(np.asarray(tokens, dtype=np.int32), 0, bt, self.dummy_slot, [])], out)
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

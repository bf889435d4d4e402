"""What the serving engines share: the decode half of the scheduler's decoder interface (batched steps,
windows of greedy steps fed back on the device, one replayed CUDA graph per padded batch size), device
error checks, host-side fault injection and time accounting.

A subclass provides ``_decode_steps(tok, pos, bts, window, greedy, slots)`` over device tensors and sets
``device``, ``cuda``, ``block_size``, ``num_blocks``, ``max_blocks``, ``dummy_block``.  Engines with
recurrent state also set ``state_slots`` (slots the scheduler hands out) and ``dummy_slot``."""
from __future__ import annotations

import time

import numpy as np
import torch

from ..ops import _cuda


class PagedEngineBase:
    #: recurrent-state slots the scheduler hands out to running sequences (0: no recurrent state)
    state_slots = 0
    dummy_slot = 0

    def _init_common(self, cuda_graphs: bool) -> None:
        self.steps = 0
        self.cuda_graphs = bool(cuda_graphs) and self.cuda
        #: host-side fault-injection point: called with "prefill" / "decode" before the device work
        #: of that call is issued; raising from it models a failed launch without touching the GPU
        self.fault_hook = None
        self._graphs = {}
        self.graph_replays = 0
        #: host wall time spent inside prefill / decode calls (each ends with a device-to-host read,
        #: so it covers the device work) and what they processed; a serving run reports the split
        self.acct = {"prefill_s": 0.0, "prefill_calls": 0, "prefill_tokens": 0, "prefill_seqs": 0,
                     "decode_s": 0.0, "decode_calls": 0, "decode_rows": 0, "mixed_s": 0.0, "mixed_calls": 0}

    def kv_pool_capacity_tokens(self) -> int:
        return self.num_blocks * self.block_size

    def check_device(self) -> None:
        """Raise if a kernel of the step just read back reported a bounded-wait timeout (the
        scheduler calls this once per step, after the token read-back, before it commits)."""
        if self.device.type == "cuda":
            _cuda.check_error()

    @torch.no_grad()
    def decode(self, tokens: np.ndarray, positions: np.ndarray, block_tables: np.ndarray,
               window: int = 1, greedy: bool = True, slots=None):
        """One batched decode call: ``window`` on-device greedy steps (window > 1 requires greedy).
        ``slots``: the sequences' recurrent-state slots (engines with state).
        Returns (tokens [B][window], per-row top-k candidate lists or None)."""
        if self.fault_hook is not None:
            self.fault_hook("decode")
        B = int(tokens.shape[0])
        t0 = time.perf_counter()
        try:
            return self._decode(tokens, positions, block_tables, window, greedy, slots)
        finally:
            a = self.acct
            a["decode_s"] += time.perf_counter() - t0
            a["decode_calls"] += 1
            a["decode_rows"] += B * window

    def _decode(self, tokens, positions, block_tables, window, greedy, slots):
        dev = self.device
        if self.cuda_graphs and (greedy or window > 1):
            out = self._decode_graphed(tokens, positions, block_tables, window, slots)
            return [row.tolist() for row in out], None
        tok = torch.from_numpy(np.ascontiguousarray(tokens)).to(dev)
        pos = torch.from_numpy(np.ascontiguousarray(positions)).to(dev)
        bts = torch.from_numpy(np.ascontiguousarray(block_tables)).to(dev)
        sl = torch.from_numpy(np.ascontiguousarray(slots, dtype=np.int32)).to(dev) if self.state_slots else None
        out_t, topks = self._decode_steps(tok, pos, bts, window, greedy or window > 1, sl)
        out = out_t.cpu().numpy()
        cand = None
        if topks is not None:
            idx, vals = topks[0].cpu().tolist(), topks[1].cpu().tolist()
            cand = [list(zip(i, v)) for i, v in zip(idx, vals)]
        return [row.tolist() for row in out], cand

    # ---- CUDA-graph decode: one captured graph per (padded batch, window)
    @staticmethod
    def _bucket(b: int) -> int:
        for cap in (1, 2, 4, 8, 16, 24, 32, 48, 64, 96, 128, 160, 192, 224, 256):
            if b <= cap:
                return cap
        return -(-b // 64) * 64

    def _decode_graphed(self, tokens, positions, block_tables, window: int, slots=None):
        """Greedy decode through a replayed CUDA graph.  The batch is padded to a bucket size with
        rows that sit at position 0 of the dummy block (and the dummy slot); inputs travel through
        pinned staging."""
        B = int(tokens.shape[0])
        Bp = self._bucket(B)
        key = (Bp, window)
        g = self._graphs.get(key)
        if g is None:
            g = self._capture(Bp, window)
            self._graphs[key] = g
        h_tok, h_pos, h_bts, h_slot = g["h_tok"], g["h_pos"], g["h_bts"], g["h_slot"]
        h_tok[:B] = torch.from_numpy(np.ascontiguousarray(tokens, dtype=np.int32))
        h_pos[:B] = torch.from_numpy(np.ascontiguousarray(positions, dtype=np.int32))
        h_bts[:B] = torch.from_numpy(np.ascontiguousarray(block_tables, dtype=np.int32))
        if self.state_slots:
            h_slot[:B] = torch.from_numpy(np.ascontiguousarray(slots, dtype=np.int32))
        if Bp > B:
            h_tok[B:] = 0
            h_pos[B:] = 0
            h_bts[B:] = self.dummy_block
            h_slot[B:] = self.dummy_slot
        g["tok"].copy_(h_tok, non_blocking=True)
        g["pos"].copy_(h_pos, non_blocking=True)
        g["bts"].copy_(h_bts, non_blocking=True)
        if self.state_slots:
            g["slot"].copy_(h_slot, non_blocking=True)
        g["graph"].replay()
        self.graph_replays += 1
        self.steps += window
        g["h_out"].copy_(g["out"], non_blocking=True)
        torch.cuda.current_stream().synchronize()
        return g["h_out"][:B].numpy().copy()

    def _capture(self, Bp: int, window: int):
        dev = self.device
        mb = self.max_blocks
        g = {"tok": torch.zeros(Bp, device=dev, dtype=torch.int32),
             "pos": torch.zeros(Bp, device=dev, dtype=torch.int32),
             "bts": torch.full((Bp, mb), self.dummy_block, device=dev, dtype=torch.int32),
             "slot": torch.full((Bp,), self.dummy_slot, device=dev, dtype=torch.int32),
             "h_tok": torch.zeros(Bp, dtype=torch.int32).pin_memory(),
             "h_pos": torch.zeros(Bp, dtype=torch.int32).pin_memory(),
             "h_bts": torch.zeros(Bp, mb, dtype=torch.int32).pin_memory(),
             "h_slot": torch.zeros(Bp, dtype=torch.int32).pin_memory(),
             "h_out": torch.zeros(Bp, window, dtype=torch.int32).pin_memory()}
        steps0 = self.steps
        slot = g["slot"] if self.state_slots else None
        # warm-up on a side stream (lazy one-time setup such as kernel attributes and symmetric
        # buffers must not happen during capture), then capture the same work
        side = torch.cuda.Stream(device=dev)
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            for _ in range(2):
                self._decode_steps(g["tok"], g["pos"], g["bts"], window, True, slot)
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        # thread-local capture mode: other threads of the process (e.g. a process group's watchdog)
        # keep making CUDA calls of their own while this thread captures
        with torch.cuda.graph(graph, capture_error_mode="thread_local"):
            out, _ = self._decode_steps(g["tok"], g["pos"], g["bts"], window, True, slot)
        g["graph"], g["out"] = graph, out
        self.steps = steps0
        return g

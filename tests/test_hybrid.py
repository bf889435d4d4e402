"""Hybrid decoders without a GPU: configuration, checkpoints, state slots in the scheduler, command line,
and the tests' own oracle (its mechanisms against closed forms, and mistakes planted in it that the GPU
tests' inputs must make visible)."""
import json
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_oracle as oracle  # noqa: E402
import hybrid_util as hu  # noqa: E402
from hybrid_util import attn, glu, mamba  # noqa: E402

from brain_b200.checkpoint import st  # noqa: E402
from brain_b200.models import build_from_config  # noqa: E402
from brain_b200.models.config import HybridConfig, config_from_json  # noqa: E402
from brain_b200.serve.paged import BlockAllocator, CachedSequence, StateSlots  # noqa: E402
from brain_b200.serve.scheduler import Scheduler  # noqa: E402


def test_config_round_trip_and_registry():
    m, _, cfg = hu.mixed_model()
    again = config_from_json(json.dumps(cfg))
    assert isinstance(again, HybridConfig) and again.to_json() == cfg
    assert cfg["layers"][1]["mlp"] is None and "rot" not in cfg["layers"][4]["mixer"]
    assert build_from_config(cfg).cfg == m.cfg
    assert m.cfg.param_count() == sum(t.numel() for t in m.reference_state().values())
    from brain_b200 import arch
    assert arch.by_id("pakalix").family == "hybrid"


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=15),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=42),
    lambda c: c["layers"][0]["mixer"].update(groups=4),
    lambda c: c["layers"][0]["mixer"].update(norm_groups=5),
    lambda c: c["layers"][0]["mixer"].update(conv=0),
    lambda c: c["layers"][0].update(type="ring"),
    lambda c: c["layers"][0]["mlp"].update(kind="routed"),
    lambda c: c["layers"][1]["mixer"].update(vdim=8),
    lambda c: c.update(architecture="Unheard-of"),
    lambda c: c.update(layers=[]),
])
def test_config_errors_are_reported(change):
    _, _, cfg = hu.mixed_model()
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    with pytest.raises(ValueError):
        config_from_json(cfg)


def test_checkpoint_directory_and_file(tmp_path):
    m, _, cfg = hu.mixed_model()
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    specs = [(n, s, "BF16") for n, s in m.cfg.tensors()]
    w = st.StWriter(str(tmp_path / "model.safetensors"), specs, {})
    for n, _, _ in specs:
        w.write(n, m.tensor(n))
    w.close()
    from brain_b200.cli.main import main
    out = str(tmp_path / "one.safetensors")
    assert main(["pakalix", "import", str(tmp_path), "--out", out]) == 0
    for src in (str(tmp_path), out):
        again, _, _ = st.load_model(src)
        for n, t in m.reference_state().items():
            assert torch.equal(again.tensor(n), t), n
    # a tensor of another size, and a missing one, are errors
    bad = dict(m.reference_state())
    bad["head"] = bad["head"][:-1]
    with pytest.raises(ValueError):
        build_from_config(cfg).load_reference_state(bad)
    del bad["head"]
    with pytest.raises(KeyError):
        build_from_config(cfg).load_reference_state(bad)


def test_import_into_the_store(tmp_path, capsys):
    m, _, cfg = hu.mixed_model()
    src = str(tmp_path / "m.safetensors")
    st.save_model(src, m, dtype="BF16")
    from brain_b200.cli.main import main
    assert main(["import", "pakalix", src, "--id", "local/tiny", "--models-dir", str(tmp_path / "store")]) == 0
    from brain_b200.modelref import ModelRef
    from brain_b200.modelstore import Store
    lm = Store(str(tmp_path / "store")).local(ModelRef.parse("local/tiny"))
    assert lm is not None and lm.card.family == "hybrid"
    assert main(["pakalix"]) == 2 and main(["pakalix", "infer"]) == 2
    if not torch.cuda.is_available():
        assert main(["pakalix", "infer", "--model", src, "--tokens", "1,2,3"]) == 1


def test_engine_refuses_the_cpu():
    from brain_b200.ops._cuda import NativeError
    from brain_b200.serve.engine import make_engine
    with pytest.raises(NativeError):
        make_engine(hu.mixed_model()[0], device="cpu")


# ------------------------------------------------------------------------------------ slots
def test_state_slots_and_cached_sequences():
    s = StateSlots(2)
    a, b = s.alloc(), s.alloc()
    assert {a, b} == {0, 1} and s.available() == 0
    with pytest.raises(MemoryError):
        s.alloc()
    s.release(a)
    with pytest.raises(RuntimeError):
        s.release(a)
    assert s.alloc() == a
    s.release(a)
    s.release(b)
    alloc = BlockAllocator(4, 4)
    q = CachedSequence(alloc, s, 4)
    assert q.extend(3)[0] == 0
    start, table = q.extend(6)
    assert start == 3 and alloc.free_blocks() == 1 and len(set(table[:3].tolist())) == 3
    with pytest.raises(MemoryError):
        q.extend(9)
    q.release()
    assert alloc.free_blocks() == 4 and s.available() == 2


class SlotDecoder:
    """Keeps a running sum per slot, as a recurrent model keeps its state: a lost, shared or swapped slot
    changes the tokens."""
    vocab, block_size, num_blocks = 50, 4, 64
    max_prefill_tokens, max_seq_len, topk_capacity = 8, 64, 8

    def __init__(self, slots):
        self.state_slots = slots
        self.sum = [0] * slots
        self.in_use = set()

    def prefill_chunk(self, tokens, start, bt, last, greedy, slot):
        if start == 0:
            self.sum[slot] = 0
        self.sum[slot] += int(tokens.sum())
        return (self.sum[slot] % self.vocab, None) if last else (None, None)

    def prefill_batch(self, items):
        assert len({it[5] for it in items}) == len(items)
        return [self.prefill_chunk(*it) for it in items]

    def decode(self, tokens, positions, bts, window, greedy, slots):
        assert len(set(slots.tolist())) == len(slots) and slots.min() >= 0
        out = []
        for t, s in zip(tokens, slots):
            row, cur = [], int(t)
            for _ in range(window):
                self.sum[s] += cur
                cur = self.sum[s] % self.vocab
                row.append(cur)
            out.append(row)
        return out, None


@pytest.mark.parametrize("slots,window", [(2, 1), (3, 4), (8, 4)])
def test_scheduler_hands_out_slots(slots, window):
    dec = SlotDecoder(slots)
    sched = Scheduler(dec, max_batch=4, window=window)
    rng = np.random.default_rng(0)
    prompts = [rng.integers(1, 50, int(n)).tolist() for n in rng.integers(1, 30, 12)]
    prompts[5] = prompts[4]              # an equal prompt must not adopt cached pages: its state is its own
    ids = [sched.submit(p, 7) for p in prompts]
    for i in range(400):
        if sched.is_idle():
            break
        sched.step()
        if i == 4:
            sched.cancel(ids[3])
    for k, (rid, p) in enumerate(zip(ids, prompts)):
        if k == 3:
            continue
        total, want = sum(p), []
        cur = total % 50
        for _ in range(7):
            want.append(cur)
            total += cur
            cur = total % 50
        assert sched.tokens_of(rid) == want, k
    from brain_b200 import _host
    assert _host.lib().bbh_sched_free_slots(sched._h) == slots
    assert sched.stats()["free_blocks"] == dec.num_blocks and sched.stats()["kv_prefix_hit_tokens"] == 0


def test_speculative_decoding_is_refused():
    from brain_b200.serve.spec import ngram_draft, spec_decode
    with pytest.raises(ValueError):
        spec_decode(SlotDecoder(2), [1, 2, 3], 4, 2, ngram_draft(2))


# ------------------------------------------------------------------------------------ the oracle itself
def test_oracle_mechanisms_against_closed_forms():
    rng = np.random.default_rng(1)
    u, w, b = rng.standard_normal((9, 3)), rng.standard_normal((3, 4)), rng.standard_normal(3)
    ref = torch.nn.functional.conv1d(torch.tensor(u.T)[None], torch.tensor(w)[:, None], torch.tensor(b), padding=3,
                                     groups=3)[0, :, :9].T.numpy()
    assert np.allclose(oracle.causal_conv(u, w, b), ref)
    # without decay and with unit steps the state is a running sum of outer products
    x, B, C = rng.standard_normal((5, 2, 3)), rng.standard_normal((5, 1, 4)), rng.standard_normal((5, 1, 4))
    y, S = oracle.state_space(x, B, C, np.ones((5, 2)), np.full(2, -np.inf), np.zeros(2))
    assert np.allclose(S[1], sum(np.outer(B[t, 0], x[t, 1]) for t in range(5)))
    assert np.allclose(y[4, 0], S[0].T @ C[4, 0])
    # a portion carried on from its predecessor's state is the whole
    dt, A, D = rng.random((5, 2)), rng.standard_normal(2), rng.standard_normal(2)
    y, S = oracle.state_space(x, B, C, dt, A, D)
    y1, S1 = oracle.state_space(x[:2], B[:2], C[:2], dt[:2], A, D)
    y2, S2 = oracle.state_space(x[2:], B[2:], C[2:], dt[2:], A, D, S1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S2, S)
    q = rng.standard_normal((4, 2, 8))
    r = oracle.rotate(q, np.arange(4.0), 6, 100.0)
    assert np.allclose(r[0], q[0]) and np.allclose(r[:, :, 6:], q[:, :, 6:])
    assert np.allclose((r ** 2).sum(-1), (q ** 2).sum(-1)) and not np.allclose(r[1], q[1])
    k = rng.standard_normal((4, 1, 8))
    v = rng.standard_normal((4, 1, 5))
    o = oracle.attend(q, k, v, 0.4, None)
    ref = torch.nn.functional.scaled_dot_product_attention(
        *(torch.tensor(t).permute(1, 0, 2) for t in (q, np.repeat(k, 2, 1), np.repeat(v, 2, 1))), is_causal=True,
        scale=0.4).permute(1, 0, 2).numpy()
    assert np.allclose(o, ref)
    assert np.allclose(oracle.attend(q, k, v, 0.4, 1e6), ref, atol=1e-6)


PLANTED = {
    "softcap left out": ("attend", lambda f: lambda q, k, v, s, c: f(q, k, v, s, None)),
    "one key too few": ("attend", lambda f: lambda q, k, v, s, c: f(q, np.concatenate([k[:1], k[:-1]]), v, s, c)),
    "rotation by interleaved pairs": ("rotate", lambda f: lambda x, p, d, b: x[:, :, ::-1]),
    "rotation of one position more": ("rotate", lambda f: lambda x, p, d, b: f(x, p * 1.05, d, b)),
    "gate after the norm": ("gated_group_norm", lambda f: lambda y, z, w, g, e: oracle.rms(
        y.reshape(len(y), g, -1), e).reshape(y.shape) * w * oracle.silu(z)),
    "one norm group": ("gated_group_norm", lambda f: lambda y, z, w, g, e: f(y, z, w, 1, e)),
    "a lost tap": ("causal_conv", lambda f: lambda u, w, b: f(u, np.concatenate([0 * w[:, :1], w[:, 1:]], 1), b)),
    "a lost state": ("state_space", lambda f: lambda x, B, C, dt, A, D: (np.concatenate(
        [f(x[:60], B[:60], C[:60], dt[:60], A, D)[0], f(x[60:], B[60:], C[60:], dt[60:], A, D)[0]]), None)),
    "no clamp": ("clamped_glu", lambda f: lambda h, W, p, limit: f(h, W, p, 1e9)),
}


@pytest.mark.parametrize("name", sorted(PLANTED))
def test_planted_mistakes_show(name, monkeypatch):
    """The inputs of the GPU tests (this model, random tokens) turn each mistake into an error well above
    what those tests allow in bf16."""
    _, W, cfg = hu.mixed_model(sharp=3.0)
    toks = hu.tokens(150, 211, 4)
    want = oracle.forward(cfg, W, toks)
    fn, wrap = PLANTED[name]
    monkeypatch.setattr(oracle, fn, wrap(getattr(oracle, fn)))
    assert hu.error(oracle.forward(cfg, W, toks), want) > 1.5 * hu.TOL["bf16"]

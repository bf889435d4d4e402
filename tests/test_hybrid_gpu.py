"""Hybrid decoders on the GPU against the plain numpy restatement: each mechanism alone, prompts against
token-by-token decoding, portions, batches, reuse of pages and slots, long decoding, and greedy generation
through the scheduler."""
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_oracle as oracle  # noqa: E402
import hybrid_util as hu  # noqa: E402
from hybrid_util import TOL, attn, glu, mamba  # noqa: E402

pytestmark = pytest.mark.gpu

MECHANISMS = {
    "attention": [(attn(), None), (attn(), None)],
    "attention_plain": [(attn(rot=0, softcap=None, v_mix=False), None)],
    "attention_one_kv_head": [(attn(heads=8, kv_heads=1, dim=32, vdim=48, rot=32), glu())],
    "attention_no_groups": [(attn(heads=5, kv_heads=5, dim=20, vdim=12, rot=6), None)],
    "attention_wide": [(attn(heads=4, kv_heads=2, dim=104, vdim=120, rot=64), None)],
    "attention_wide_keys": [(attn(heads=4, kv_heads=4, dim=96, vdim=16, rot=96), None)],
    "attention_very_wide": [(attn(heads=2, kv_heads=1, dim=160, vdim=136, rot=32), None)],
    "attention_huge": [(attn(heads=2, kv_heads=2, dim=320, vdim=264, rot=64), None)],
    "attention_low_cap": [(attn(softcap=2.0, scale=1.0), None)],
    "attention_many_shared": [(attn(heads=14, kv_heads=2, dim=8, vdim=8, rot=2), None)],
    "v_mix_skips_a_layer": [(attn(v_mix=False, vdim=16), None), (attn(), None), (attn(dim=16), glu()), (attn(), None)],
    "mamba": [(mamba(), None)],
    "mamba_one_head": [(mamba(heads=1, vdim=64, state=16, groups=1, norm_groups=1), glu())],
    "mamba_groups": [(mamba(heads=8, vdim=8, state=8, groups=4, norm_groups=16), None)],
    "mamba_odd": [(mamba(heads=3, vdim=10, state=7, groups=3, conv=5, norm_groups=2), glu(37, 0.5))],
    "mamba_no_taps": [(mamba(conv=1), None)],
    "mamba_two_taps": [(mamba(conv=2, norm_groups=1), None)],
    "mamba_wide": [(mamba(heads=2, vdim=128, state=128, groups=1, norm_groups=2), None)],
    "mamba_tall": [(mamba(heads=2, vdim=48, state=200, groups=2, norm_groups=1), None)],
    "mamba_real": [(mamba(heads=4, vdim=64, state=128, groups=1, norm_groups=1), glu(200, 3.0))],
    "mamba_half": [(mamba(heads=4, vdim=32, state=64, groups=2, norm_groups=4), None)],
}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism(name, dtype):
    m, W, cfg = hu.make(MECHANISMS[name], sharp=2.0)
    toks = hu.tokens(150, m.cfg.vocab, 1)
    want = oracle.forward(cfg, W, toks)
    s = hu.session(m, dtype)
    assert hu.error(hu.feed(s, "a", toks, [150]), want) < TOL[dtype]
    # the same through the cache: a portion, then one by one, in the pages and the slot just given back
    assert hu.error(hu.feed(s, "b", toks, [120, 1]), want) < TOL[dtype]


@pytest.mark.parametrize("width,vocab", [(100, 203), (36, 64), (328, 1000)])
def test_sizes_that_need_padding(width, vocab):
    m, W, cfg = hu.mixed_model(width=width, vocab=vocab, mult=1.0)
    toks = hu.tokens(70, vocab, 2)
    want = oracle.forward(cfg, W, toks)
    for dtype in ("fp32", "bf16"):
        assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, [33, 1, 20, 2, 1]), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_residual_stream_after_every_layer(dtype):
    m, W, cfg = hu.mixed_model()
    toks, layers = hu.tokens(40, m.cfg.vocab, 3), []
    oracle.forward(cfg, W, toks, layers)
    got = hu.engine(m, dtype).residual_trace(toks).cpu().numpy()
    for i, want in enumerate(layers):
        assert np.abs(got[i] - want).max() < (2e-5 if dtype == "fp32" else 0.06) * np.abs(want).max(), i


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("sizes", [[300], [1], [2], [3], [5, 2, 17, 64, 1, 2], [15, 1, 16, 2, 31, 127, 1], [129, 128]])
def test_portions_do_not_matter(sizes, dtype):
    m, W, cfg = hu.mixed_model(sharp=3.0)
    toks = hu.tokens(300, m.cfg.vocab, 4)
    want = oracle.forward(cfg, W, toks)
    assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, sizes), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_batches_of_unequal_requests(dtype):
    """Portions of some requests beside single tokens of others, requests left out of steps, pages and
    slots given back and used again; each request as if it were alone."""
    m, W, cfg = hu.mixed_model(sharp=2.0)
    s = hu.session(m, dtype, num_blocks=30)
    rng = np.random.default_rng(5)
    todo = [(f"r{i}", hu.tokens(int(n), m.cfg.vocab, 100 + i)) for i, n in enumerate([130, 1, 47, 2, 90, 33, 118, 16, 3, 64])]
    want = {r: oracle.forward(cfg, W, t) for r, t in todo}
    got, live = {r: [] for r, _ in todo}, {}
    while todo or live:
        while todo and len(live) < 4 and sum(-(-len(t) // 64) * 4 for t, _ in live.values()) + -(-len(todo[0][1]) // 64) * 4 <= 30:
            r, t = todo.pop(0)
            live[r] = (t, 0)
        step = []
        for r, (t, at) in live.items():
            if len(live) > 1 and rng.random() < 0.2:
                continue
            n = 1 if at and rng.random() < 0.5 else int(rng.integers(1, 40))
            step.append((r, t[at:at + n], list(range(min(n, len(t) - at)))))
        if not step:
            continue
        out = s.step(step)
        i = 0
        for r, part, _ in step:
            got[r].append(out[i:i + len(part)])
            i += len(part)
            t, at = live[r]
            live[r] = (t, at + len(part))
            if live[r][1] == len(t):
                s.end(r)
                del live[r]
    for r in want:
        assert hu.error(np.concatenate(got[r]), want[r]) < TOL[dtype], r
    assert s.alloc.free_blocks() == 30 and s.slots.available() == 4


def test_wanted_rows_come_in_request_order():
    m, W, cfg = hu.mixed_model()
    s = hu.session(m, "fp32")
    a, b, c = (hu.tokens(n, m.cfg.vocab, n) for n in (20, 30, 25))
    s.step([("a", a[:10], []), ("b", b[:29], [28])])
    out = s.step([("a", a[10:11], [0]), ("c", c, [24, 3]), ("b", b[29:], [0])])
    wa, wb, wc = (oracle.forward(cfg, W, t) for t in (a[:11], b, c))
    assert hu.error(out, np.stack([wa[10], wc[24], wc[3], wb[29]])) < TOL["fp32"]
    assert s.step([("a", a[11:13], [])]) is None


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_long_decoding(dtype):
    m, W, cfg = hu.mixed_model(sharp=2.0)
    toks = hu.tokens(600, m.cfg.vocab, 6)
    want = oracle.forward(cfg, W, toks)
    assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, [9, 1]), want) < TOL[dtype]


def test_stale_pages_and_slots_do_not_leak():
    """A request whose pages and slot hold another request's values (NaNs at their places that are not
    written again would show too) gives the logits of a fresh engine, bit for bit."""
    m, _, _ = hu.mixed_model()
    t1, t2 = hu.tokens(200, m.cfg.vocab, 7), hu.tokens(90, m.cfg.vocab, 8)
    fresh = hu.feed(hu.session(m, "bf16"), "x", t2, [50, 1, 7])
    s = hu.session(m, "bf16")
    hu.feed(s, "a", t1, [200])
    assert np.array_equal(hu.feed(s, "b", t2, [50, 1, 7]), fresh)


def test_a_step_that_cannot_be_run_is_refused_on_the_host():
    m, _, _ = hu.mixed_model()
    s = hu.session(m, "bf16")
    with pytest.raises(ValueError):
        s.step([("a", [m.cfg.vocab], [0])])
    with pytest.raises(ValueError):
        s.step([("b", [1, 2], [2])])
    with pytest.raises(MemoryError):
        s.step([("c", [1] * 700, [])])
    from brain_b200.serve.engine import make_engine
    for bad in (dict(weights="int8"), dict(kv_dtype="int8"), dict(dtype="fp8")):
        with pytest.raises(ValueError):
            make_engine(m, device="cuda:0", **bad)


# ------------------------------------------------------------------------------------ generation
def _oracle_greedy(cfg, W, prompt, n):
    toks = list(prompt)
    margin = np.inf
    for _ in range(n):
        lg = np.sort(oracle.forward(cfg, W, toks)[-1])
        margin = min(margin, lg[-1] - lg[-2])
        toks.append(int(np.argmax(oracle.forward(cfg, W, toks)[-1])))
    return toks[len(prompt):], margin


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("mixed", [True, False])
def test_greedy_generation_through_the_scheduler(mixed, graphs):
    from brain_b200.serve.scheduler import Scheduler
    m, W, cfg = hu.mixed_model(vocab=97)
    eng = hu.engine(m, "fp32", num_blocks=24, max_prefill=32, state_slots=3, cuda_graphs=graphs)
    sched = Scheduler(eng, max_batch=3, window=4, mixed=mixed)
    prompts = [hu.tokens(n, 97, 50 + n) for n in (70, 1, 33, 5, 64, 2)]
    ids = [sched.submit(p, 9) for p in prompts]
    sched.run_until_idle()
    for rid, p in zip(ids, prompts):
        want, margin = _oracle_greedy(cfg, W, p, 9)
        if margin > 1e-3:
            assert sched.tokens_of(rid) == want, len(p)
    st = sched.stats()
    assert st["free_blocks"] == 24 and st["prefix_entries"] == 0
    assert bool(eng.graph_replays) == graphs


def test_sampling_and_cancel_through_the_scheduler():
    from brain_b200.serve.sampling import SampleParams
    from brain_b200.serve.scheduler import Scheduler
    m, _, _ = hu.mixed_model(vocab=97)

    def run(cancel):
        eng = hu.engine(m, "bf16", state_slots=2)
        sched = Scheduler(eng, max_batch=2, mixed=True)
        a = sched.submit(hu.tokens(20, 97, 1), 12, SampleParams(0.9, 20, 0.95), seed=5)
        b = sched.submit(hu.tokens(30, 97, 2), 30)
        c = sched.submit(hu.tokens(40, 97, 3), 12, SampleParams(0.7, 0, 1.0), seed=6)
        for _ in range(3):
            sched.step()
        if cancel:
            sched.cancel(b)
        sched.run_until_idle()
        return sched.tokens_of(a), sched.tokens_of(c)

    alone, other = run(False), run(True)
    assert len(alone[0]) == 12 and alone == other


def test_serve_prompts_entry_point():
    from brain_b200.serve.offline import serve_prompts
    m, W, cfg = hu.mixed_model(vocab=97)
    prompts = [hu.tokens(n, 97, 80 + n) for n in (17, 40)]
    r = serve_prompts(m.to("cuda:0"), prompts, max_new=6)
    assert [len(o) for o in r["outputs"]] == [6, 6]
    m32 = serve_prompts(m, prompts, max_new=6, dtype="fp32")
    for p, o in zip(prompts, m32["outputs"]):
        want, margin = _oracle_greedy(cfg, W, p, 6)
        if margin > 1e-3:
            assert o == want

"""Zepesun decoders on the GPU against the plain numpy restatement: each mechanism alone, prompts against
token-by-token decoding, portions, batches, reuse of pages and slots, long decoding, and greedy generation
through the scheduler."""
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_util as hu  # noqa: E402
import zepesun_oracle as oracle  # noqa: E402
import zepesun_util as zu  # noqa: E402
from hybrid_util import TOL  # noqa: E402
from zepesun_util import attn, both, gelu, latent, memory, moe  # noqa: E402

pytestmark = pytest.mark.gpu

MECHANISMS = {
    "latent": [(latent(), None)],
    "latent_one_head": [(latent(heads=1, dim=64, rot=64, vdim=128, kv_rank=128), None)],
    "latent_many_heads": [(latent(heads=40, dim=8, rot=8, vdim=8, kv_rank=72), None)],
    "latent_odd": [(latent(heads=3, dim=13, rot=6, vdim=11, kv_rank=29), None)],
    "latent_wide_heads": [(latent(heads=2, dim=128, rot=64, vdim=128, kv_rank=96), None)],
    "latent_wide_rank": [(latent(heads=2, dim=32, rot=64, vdim=32, kv_rank=512), None)],
    "memory": [(memory(), None)],
    "memory_small": [(memory(heads=5, dim=8, vdim=8), None)],
    "memory_keys_wide": [(memory(heads=2, dim=96, vdim=32), None)],
    "memory_values_wide": [(memory(heads=2, dim=32, vdim=96), None)],
    "memory_both_wide": [(memory(heads=1, dim=128, vdim=128, cap=5.0), None)],
    "memory_odd": [(memory(heads=3, dim=21, vdim=37), None)],
    "memory_beyond_tiles": [(memory(heads=1, dim=40, vdim=200), None)],
    "memory_beyond_tiles_keys": [(memory(heads=2, dim=136, vdim=9), None)],
    "memory_tight_gates": [(memory(cap=0.3), None)],
    "memory_wide_gates": [(memory(cap=30.0), None)],
    "both": [(both(), None)],
    "both_itself_only": [(both(attn(window=1)), None)],
    "both_two_keys": [(both(attn(window=2)), None), (both(attn(window=3)), None)],
    "both_every_key": [(both(attn(window=None)), None)],
    "both_wide_window": [(both(attn(window=129)), None)],
    "both_one_kv_head": [(both(attn(5, 1, 16, 72)), None)],
    "both_as_many_kv_heads": [(both(attn(3, 3, 72, 16)), None)],
    "both_odd": [(both(attn(6, 2, 21, 13), memory(2, 11, 19)), None)],
    "both_wide_heads": [(both(attn(2, 1, 136, 160, 0.1)), None)],
    "both_factors": [(both(ls=0.1, rs=2.5), None)],
    "dense": [(memory(), gelu(200)), (memory(), gelu(17))],
    "moe": [(memory(), moe())],
    "moe_no_groups": [(memory(), moe(groups=1, keep=1))],
    "moe_every_group": [(memory(), moe(groups=4, keep=4))],
    "moe_one_expert_each": [(memory(), moe(top=1, scale=1.0, shared=None))],
    "moe_all_experts": [(memory(), moe(experts=4, top=4, groups=1, keep=1))],
    "moe_groups_of_one": [(memory(), moe(experts=6, top=2, groups=6, keep=3))],
    "moe_one_expert": [(memory(), moe(experts=1, top=1, groups=1, keep=1))],
    "moe_many": [(memory(), moe(ff=8, experts=72, top=8, groups=8, keep=4))],
    "moe_more": [(memory(), moe(ff=5, experts=160, top=5, groups=2, keep=1, shared=(9, 0.7)))],
}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism(name, dtype):
    m, W, cfg = zu.make(MECHANISMS[name], sharp=2.0)
    toks = hu.tokens(150, m.cfg.vocab, 1)
    want = oracle.forward(cfg, W, toks)
    s = hu.session(m, dtype)
    assert hu.error(hu.feed(s, "a", toks, [150]), want) < TOL[dtype]
    # the same through the cache: a portion, then one by one, in the pages and the slot just given back
    assert hu.error(hu.feed(s, "b", toks, [120, 1]), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_normaliser_shows(dtype):
    """The heads' norm takes a common factor off; with a large epsilon the floor under the normaliser counts."""
    m, W, cfg = zu.make([(memory(heads=3, dim=16, vdim=24), None), (both(), None)], eps=0.02)
    toks = hu.tokens(150, m.cfg.vocab, 9)
    want = oracle.forward(cfg, W, toks)
    for sizes in ([150], [70, 3, 1]):
        assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, sizes), want) < TOL[dtype]


@pytest.mark.parametrize("width,vocab", [(100, 203), (36, 64), (328, 1000)])
def test_sizes_that_need_padding(width, vocab):
    m, W, cfg = zu.mixed_model(width=width, vocab=vocab)
    toks = hu.tokens(70, vocab, 2)
    want = oracle.forward(cfg, W, toks)
    for dtype in ("fp32", "bf16"):
        assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, [33, 1, 20, 2, 1]), want) < TOL[dtype]


def test_rows_wider_than_a_block_keeps():
    m, W, cfg = zu.make([(memory(), moe(ff=8)), (memory(), gelu(24))], width=4104, vocab=64)
    toks = hu.tokens(20, 64, 2)
    want = oracle.forward(cfg, W, toks)
    for dtype in ("fp32", "bf16"):
        assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, [9, 1, 2]), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_residual_stream_after_every_layer(dtype):
    m, W, cfg = zu.mixed_model()
    toks, layers = hu.tokens(40, m.cfg.vocab, 3), []
    oracle.forward(cfg, W, toks, layers)
    got = hu.engine(m, dtype).residual_trace(toks).cpu().numpy()
    for i, want in enumerate(layers):
        assert np.abs(got[i] - want).max() < (2e-5 if dtype == "fp32" else 0.06) * np.abs(want).max(), i


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("sizes", [[300], [1], [2], [3], [5, 2, 17, 64, 1, 2], [15, 1, 16, 2, 31, 127, 1], [129, 128]])
def test_portions_do_not_matter(sizes, dtype):
    m, W, cfg = zu.mixed_model(sharp=3.0)
    toks = hu.tokens(300, m.cfg.vocab, 4)
    want = oracle.forward(cfg, W, toks)
    assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, sizes), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_batches_of_unequal_requests(dtype):
    """Portions of some requests beside single tokens of others, requests left out of steps, pages and
    slots given back and used again; each request as if it were alone."""
    m, W, cfg = zu.mixed_model(sharp=2.0)
    s = hu.session(m, dtype, num_blocks=30)
    rng = np.random.default_rng(5)
    todo = [(f"r{i}", hu.tokens(int(n), m.cfg.vocab, 100 + i)) for i, n in enumerate([130, 1, 47, 2, 90, 33, 118, 16, 3, 64])]
    want = {r: oracle.forward(cfg, W, t) for r, t in todo}
    got, live = {r: [] for r, _ in todo}, {}
    pages = lambda t: -(-len(t) // 64) * 4
    while todo or live:
        while todo and len(live) < 4 and sum(pages(t) for t, _ in live.values()) + pages(todo[0][1]) <= 30:
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
        out, i = s.step(step), 0
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


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_long_decoding(dtype):
    m, W, cfg = zu.mixed_model(sharp=2.0)
    toks = hu.tokens(500, m.cfg.vocab, 6)
    want = oracle.forward(cfg, W, toks)
    assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, [9, 1]), want) < TOL[dtype]


@pytest.mark.parametrize("dtype,tol", [("fp32", 4e-5), ("bf16", 0.04)])
def test_memory_that_hardly_forgets(dtype, tol):
    """Forget gates within 1e-5 of one over a long sequence."""
    m, W, cfg = zu.make([(memory(cap=15.0), None), (both(right=memory(cap=13.0)), None)])
    for n, t in m.reference_state().items():
        if n.endswith("f.b"):
            t.fill_(24.0)
            W[n] = t.numpy().astype(np.float64)
    toks = hu.tokens(620, m.cfg.vocab, 16)
    want = oracle.forward(cfg, W, toks)
    assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, [400, 100, 1]), want) < tol


def test_stale_pages_and_slots_do_not_leak():
    """A request whose pages and slot hold another request's values gives the logits of a fresh engine, bit
    for bit."""
    m, _, _ = zu.mixed_model()
    t1, t2 = hu.tokens(200, m.cfg.vocab, 7), hu.tokens(90, m.cfg.vocab, 8)
    fresh = hu.feed(hu.session(m, "bf16"), "x", t2, [50, 1, 7])
    s = hu.session(m, "bf16")
    hu.feed(s, "a", t1, [200])
    assert np.array_equal(hu.feed(s, "b", t2, [50, 1, 7]), fresh)


def test_what_else_is_in_the_batch_does_not_matter():
    """Bit for bit within one kind of row: experts' rows land on other tiles, their values stay."""
    m, _, _ = zu.mixed_model()
    t = [hu.tokens(n, m.cfg.vocab, 30 + n) for n in (80, 33, 2)]
    s = hu.session(m, "bf16")
    alone = s.step([("a", t[0], list(range(80)))])
    s.end("a")
    together = s.step([("b", t[1], []), ("c", t[0], list(range(80))), ("d", t[2], [])])
    assert np.array_equal(alone, together)


def test_steps_that_cannot_be_run_are_refused_on_the_host():
    m, _, _ = zu.mixed_model(positions=100)
    s = hu.session(m, "bf16")
    assert s.engine.max_seq_len == 100
    with pytest.raises(ValueError):
        s.step([("a", [m.cfg.vocab], [0])])
    s = hu.session(m, "bf16")
    with pytest.raises((ValueError, MemoryError)):
        s.step([("c", [1] * 101, [])])             # no position is learned for the last of them
    with pytest.raises(ValueError):
        hu.engine(m, "bf16", kv_dtype="int8")


# ------------------------------------------------------------------------------------ generation
def _oracle_greedy(cfg, W, prompt, n):
    toks, margin = list(prompt), np.inf
    for _ in range(n):
        row = oracle.forward(cfg, W, toks)[-1]
        lg = np.sort(row)
        margin = min(margin, lg[-1] - lg[-2])
        toks.append(int(np.argmax(row)))
    return toks[len(prompt):], margin


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("mixed", [True, False])
def test_greedy_generation_through_the_scheduler(mixed, graphs):
    from brain_b200.serve.scheduler import Scheduler
    m, W, cfg = zu.mixed_model(vocab=97)
    eng = hu.engine(m, "fp32", num_blocks=24, max_prefill=32, state_slots=3, cuda_graphs=graphs)
    sched = Scheduler(eng, max_batch=3, window=4, mixed=mixed)
    prompts = [hu.tokens(n, 97, 50 + n) for n in (70, 1, 33, 5, 64, 2)]
    ids = [sched.submit(p, 9) for p in prompts]
    sched.run_until_idle()
    checked = 0
    for rid, p in zip(ids, prompts):
        want, margin = _oracle_greedy(cfg, W, p, 9)
        if margin > 1e-3:
            checked += 1
            assert sched.tokens_of(rid) == want, len(p)
    assert checked >= 4
    assert sched.stats()["free_blocks"] == 24 and bool(eng.graph_replays) == graphs


def test_bf16_graphs_equal_plain_steps():
    from brain_b200.serve.scheduler import Scheduler
    m, _, _ = zu.mixed_model(vocab=97)
    out = []
    for graphs in (True, False):
        sched = Scheduler(hu.engine(m, "bf16", num_blocks=40, state_slots=3, cuda_graphs=graphs), max_batch=3, window=4)
        ids = [sched.submit(hu.tokens(n, 97, 60 + n), 12) for n in (40, 3, 77)]
        sched.run_until_idle()
        out.append([sched.tokens_of(i) for i in ids])
    assert out[0] == out[1] and all(len(o) == 12 for o in out[0])


def test_serve_prompts_and_command_line(tmp_path, capsys):
    from brain_b200.checkpoint import st
    from brain_b200.cli.main import main
    from brain_b200.serve.offline import serve_prompts
    m, W, cfg = zu.mixed_model(vocab=97)
    prompts = [hu.tokens(n, 97, 80 + n) for n in (17, 40)]
    src = str(tmp_path / "m.safetensors")
    st.save_model(src, m, dtype="BF16")
    r = serve_prompts(m.to("cuda:0"), prompts, max_new=6, dtype="fp32")
    for p, o in zip(prompts, r["outputs"]):
        want, margin = _oracle_greedy(cfg, W, p, 6)
        assert len(o) == 6
        if margin > 1e-3:
            assert o == want
    capsys.readouterr()
    args = ["zepesun", "infer", "--model", src, "--max-new", "6", "--dtype", "fp32", "--tokens", ",".join(map(str, prompts[0]))]
    assert main(args) == 0
    assert [int(t) for t in capsys.readouterr().out.strip().split(",")] == r["outputs"][0]

"""Povipel decoders on the GPU against the plain numpy restatement: each mechanism alone, prompts against
token-by-token decoding, portions, batches, reuse of pages and slots, long decoding, and greedy generation
through the scheduler."""
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_util as hu  # noqa: E402
import povipel_oracle as oracle  # noqa: E402
import povipel_util as pu  # noqa: E402
from povipel_util import attn, both, gelu, gla, moe, ret  # noqa: E402

pytestmark = pytest.mark.gpu

#: layers, then what else the model has
MECHANISMS = {
    "both": ([(both(), None)], {}),
    "both_itself_only": ([(both(attn(window=1, pool=5)), None)], {}),
    "both_two_keys": ([(both(attn(window=2, pool=2)), None), (both(attn(window=3, pool=7)), None)], {}),
    "both_blocks_of_one": ([(both(attn(window=9, pool=1)), None)], {}),
    "both_blocks_as_wide_as_pages": ([(both(attn(window=33, pool=16)), None)], {}),
    "both_blocks_wider_than_pages": ([(both(attn(window=18, pool=37)), None)], {}),
    "both_blocks_wider_than_the_window": ([(both(attn(window=4, pool=24)), None)], {}),
    "both_many_blocks": ([(both(attn(window=3, pool=1)), None), (both(attn(window=5, pool=2)), None)], {}),
    "both_wide_window": ([(both(attn(window=129, pool=8)), None)], {}),
    "both_every_key": ([(both(attn(window=None, pool=None)), None)], {}),
    "both_no_blocks": ([(both(attn(window=17, pool=None)), None)], {}),
    "both_one_kv_head": ([(both(attn(5, 1, 16, 72, rot=16)), None)], {}),
    "both_as_many_kv_heads": ([(both(attn(3, 3, 72, 16, rot=24)), None)], {}),
    "both_odd": ([(both(attn(6, 2, 21, 14, rot=6), gla(2, 11, 19, rank=3)), None)], {}),
    "both_whole_head_rotated": ([(both(attn(2, 1, 128, 128, 0.09, rot=128)), None)], {}),
    "both_wide_heads": ([(both(attn(2, 1, 136, 160, 0.08, rot=8)), None)], {}),
    "gla_small": ([(both(right=gla(5, 8, 8)), None)], {}),
    "gla_keys_wide": ([(both(right=gla(2, 96, 32)), None)], {}),
    "gla_keys_wider": ([(both(right=gla(1, 200, 24)), None)], {}),
    "gla_keys_widest": ([(both(right=gla(1, 300, 16)), None)], {}),
    "gla_values_wide": ([(both(right=gla(2, 40, 136)), None)], {}),
    "gla_values_wider": ([(both(right=gla(1, 16, 520)), None)], {}),
    "gla_root_one": ([(both(right=gla(tau=1.0)), None)], {}),
    "gla_slow": ([(both(right=gla(tau=400.0)), None)], {}),
    "gla_many_heads": ([(both(right=gla(20, 8, 16, rank=24)), None)], {}),
    "retention": ([(ret(), None)], {}),
    "retention_both_wide": ([(ret(1, 128, 128, 128), None)], {}),
    "retention_values_wide": ([(ret(2, 32, 96, 32), None)], {}),
    "retention_beyond_tiles": ([(ret(1, 40, 200, 40), None)], {}),
    "retention_beyond_tiles_keys": ([(ret(2, 136, 9, 64), None)], {}),
    "retention_odd": ([(ret(3, 21, 37, 10), None)], {}),
    "retention_fast": ([(ret(decay=[0.01, 0.3, 1.0]), None)], {}),
    "one_stream": ([(ret(), gelu()), (both(), None)], dict(streams=1)),
    "two_streams": ([(ret(), gelu()), (both(), moe())], dict(streams=2)),
    "four_streams": ([(ret(), moe()), (both(), gelu())], dict(streams=4)),
    "seven_streams": ([(ret(), gelu()), (both(), None)], dict(streams=7)),
    "sixteen_streams": ([(ret(), gelu()), (both(), None)], dict(streams=16)),
    "looped": ([(ret(), None), (both(), gelu()), (ret(), moe())], dict(loop=(0, 2, 3))),
    "looped_alone": ([(both(), None)], dict(loop=(0, 1, 4))),
    "dense": ([(ret(), gelu(200)), (ret(), gelu(17))], {}),
    "moe": ([(ret(), moe())], {}),
    "moe_one_expert_each": ([(ret(), moe(top=1))], {}),
    "moe_all_experts": ([(ret(), moe(experts=4, top=4))], {}),
    "moe_one_expert": ([(ret(), moe(experts=1, top=1))], {}),
    "moe_many": ([(ret(), moe(ff=8, experts=72, top=8))], {}),
    "moe_more": ([(ret(), moe(ff=5, experts=160, top=3))], {}),
    "bounded_logits": ([(ret(), gelu())], dict(cap=1.5, spread=3.0)),
    "unbounded_logits": ([(ret(), gelu())], dict(cap=None)),
}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism(name, dtype):
    m, W, cfg = pu.make(MECHANISMS[name][0], sharp=2.0, **MECHANISMS[name][1])
    toks = hu.tokens(150, m.cfg.vocab, 1)
    want = oracle.forward(cfg, W, toks)
    s = hu.session(m, dtype)
    assert pu.close(hu.feed(s, "a", toks, [150]), want, dtype)
    # the same through the cache: a portion, then one by one, in the pages and the slot just given back
    assert pu.close(hu.feed(s, "b", toks, [120, 1]), want, dtype)


@pytest.mark.parametrize("width,vocab", [(100, 203), (36, 64), (328, 1000)])
def test_sizes_that_need_padding(width, vocab):
    m, W, cfg = pu.mixed_model(width=width, vocab=vocab)
    toks = hu.tokens(70, vocab, 2)
    want = oracle.forward(cfg, W, toks)
    for dtype in ("fp32", "bf16"):
        assert pu.close(hu.feed(hu.session(m, dtype), "a", toks, [33, 1, 20, 2, 1]), want, dtype)


def test_wide_rows():
    m, W, cfg = pu.make([(ret(), moe(ff=8)), (both(), gelu(24))], width=4104, vocab=64)
    toks = hu.tokens(20, 64, 2)
    want = oracle.forward(cfg, W, toks)
    for dtype in ("fp32", "bf16"):
        assert pu.close(hu.feed(hu.session(m, dtype), "a", toks, [9, 1, 2]), want, dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_residual_stream_after_every_layer(dtype):
    m, W, cfg = pu.mixed_model()
    toks, layers = hu.tokens(40, m.cfg.vocab, 3), []
    oracle.forward(cfg, W, toks, layers)
    got = hu.engine(m, dtype).residual_trace(toks).cpu().numpy()
    for i, want in enumerate(layers):
        assert np.abs(got[i] - want).max() < (2e-5 if dtype == "fp32" else 0.06) * np.abs(want).max(), i


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("sizes", [[300], [1], [2], [3], [5, 2, 17, 64, 1, 2], [15, 1, 16, 2, 31, 127, 1], [129, 128]])
def test_portions_do_not_matter(sizes, dtype):
    m, W, cfg = pu.mixed_model(sharp=2.0)
    toks = hu.tokens(300, m.cfg.vocab, 4)
    want = oracle.forward(cfg, W, toks)
    assert pu.close(hu.feed(hu.session(m, dtype), "a", toks, sizes), want, dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_batches_of_unequal_requests(dtype):
    """Portions of some requests beside single tokens of others, requests left out of steps, pages and
    slots given back and used again; each request as if it were alone."""
    m, W, cfg = pu.mixed_model(sharp=2.0)
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
        assert pu.close(np.concatenate(got[r]), want[r], dtype), r
    assert s.alloc.free_blocks() == 30 and s.slots.available() == 4


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_long_decoding(dtype):
    m, W, cfg = pu.mixed_model(sharp=2.0)
    toks = hu.tokens(500, m.cfg.vocab, 6)
    want = oracle.forward(cfg, W, toks)
    assert pu.close(hu.feed(hu.session(m, dtype), "a", toks, [9, 1]), want, dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_states_that_hardly_forget(dtype):
    """Decays within 1e-4 of one over a long sequence."""
    m, W, cfg = pu.make([(ret(decay=[0.9999, 1.0, 1.0 - 1e-5]), None), (both(right=gla(tau=64.0)), None)])
    for n, t in m.reference_state().items():
        if n.endswith("a2.b"):
            t.fill_(6.0)
            W[n] = t.numpy().astype(np.float64)
    toks = hu.tokens(620, m.cfg.vocab, 16)
    want = oracle.forward(cfg, W, toks)
    assert pu.close(hu.feed(hu.session(m, dtype), "a", toks, [400, 100, 1]), want, dtype)


@pytest.mark.parametrize("block", [16, 32, 64])
def test_page_sizes(block):
    """Pooled blocks smaller than a page, as large, larger, and across pages of every size."""
    m, W, cfg = pu.make([(both(attn(window=12, pool=p)), None) for p in (3, block, block + 5)], sharp=3.0)
    toks = hu.tokens(230, m.cfg.vocab, 18)
    want = oracle.forward(cfg, W, toks)
    for dtype in ("fp32", "bf16"):
        s = hu.session(m, dtype, block_size=block, num_blocks=640 // block)
        assert pu.close(hu.feed(s, "a", toks, [37, 1, 2, 64, 1, 1, 30]), want, dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("size,pool", pu.BORDERS)
def test_borders_of_windows_and_blocks(size, pool, dtype):
    """Every position of a sequence with loud tokens, in prompts of several cuts and decoded."""
    m, W, cfg, toks = pu.borders_model(size, pool)
    want, n = oracle.forward(cfg, W, toks), len(toks)
    for sizes in ([n], [1], [2], [size, 1], [pool, pool + 1], [n // 2, 1]):
        assert hu.error(hu.feed(hu.session(m, dtype), "a", toks, sizes), want) < hu.TOL[dtype], sizes


def test_stale_pages_and_slots_do_not_leak():
    """A request whose pages and slot hold another request's values gives the logits of a fresh engine, bit
    for bit."""
    m, _, _ = pu.mixed_model()
    t1, t2 = hu.tokens(200, m.cfg.vocab, 7), hu.tokens(90, m.cfg.vocab, 8)
    fresh = hu.feed(hu.session(m, "bf16"), "x", t2, [50, 1, 7])
    s = hu.session(m, "bf16")
    hu.feed(s, "a", t1, [200])
    assert np.array_equal(hu.feed(s, "b", t2, [50, 1, 7]), fresh)


def test_what_else_is_in_the_batch_does_not_matter():
    """Bit for bit within one kind of row: experts' rows land on other tiles, their values stay."""
    m, _, _ = pu.mixed_model()
    t = [hu.tokens(n, m.cfg.vocab, 30 + n) for n in (80, 33, 2)]
    s = hu.session(m, "bf16")
    alone = s.step([("a", t[0], list(range(80)))])
    s.end("a")
    together = s.step([("b", t[1], []), ("c", t[0], list(range(80))), ("d", t[2], [])])
    assert np.array_equal(alone, together)


def test_steps_that_cannot_be_run_are_refused_on_the_host():
    m, _, _ = pu.mixed_model()
    s = hu.session(m, "bf16", max_seq_len=96)
    with pytest.raises(ValueError):
        s.step([("a", [m.cfg.vocab], [0])])
    s = hu.session(m, "bf16", max_seq_len=96)
    with pytest.raises((ValueError, MemoryError)):
        s.step([("c", [1] * 101, [])])
    with pytest.raises(ValueError):
        hu.engine(m, "bf16", kv_dtype="int8")


def test_passes_of_a_layer_share_weights_but_not_state():
    m, _, _ = pu.mixed_model()
    e = hu.engine(m, "bf16")
    one, two = (e.layer_list[r] for r, i in enumerate(m.cfg.runs) if i == 2)
    assert one.inp.w == two.inp.w and one.kc != two.kc and one.pkc != two.pkc and one.shift_state != two.shift_state
    assert one.beside != two.beside and len({l.ssm_state for l in e.mixers if l.ssm_state}) == 7


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
    m, W, cfg = pu.mixed_model(vocab=97)
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
    m, _, _ = pu.mixed_model(vocab=97)
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
    m, W, cfg = pu.mixed_model(vocab=97)
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
    args = ["povipel", "infer", "--model", src, "--max-new", "6", "--dtype", "fp32", "--tokens", ",".join(map(str, prompts[0]))]
    assert main(args) == 0
    assert [int(t) for t in capsys.readouterr().out.strip().split(",")] == r["outputs"][0]

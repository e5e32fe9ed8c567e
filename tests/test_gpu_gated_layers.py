"""Layer-list decoders of the Teganex design on a GPU against the plain implementation in oracle/gated_layers.py (float64).
Limits as in test_gpu_layer_list.py: a few times what rounding-sized noise on every sublayer does to the oracle itself."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from oracle import gated_layers as oracle
from tests import gated_models as gm
from tests import layer_list_models as lm
from tests.test_gpu_layer_list import FLOOR, NOISE, error, run_portions

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


def model_of(c, t, dtype):
    from monoserve_b200 import registry
    from monoserve_b200.layer_list import Weights, read_config
    cfg = read_config(c, dtype)
    return registry.Model(registry._LayerList, cfg, Weights(cfg, t))


def limit_of(c, t, toks, ref, dtype):
    return max(FLOOR[dtype], 4 * error(oracle.model_logits(c, t, toks, jitter=NOISE[dtype]), ref))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(gm.MODELS))
def test_prompt_portions_and_decoding(name, dtype):
    """Whole prompts, portions down to two tokens, and token-by-token decoding give the oracle's logits; the residual after
    every layer does too (whole prompts)."""
    from monoserve_b200.session import Session
    c = gm.MODELS[name]
    t = gm.tensors(c, 11, rank=40 if name == "heads" else None)
    toks = gm.tokens(c, 75, 1)
    runs = []
    ref = oracle.model_logits(c, t, toks, runs=runs)
    limit = limit_of(c, t, toks, ref, dtype)
    with Session(model_of(c, t, dtype), max_tokens=256, page=16, keep_residual=True) as s:
        assert error(s.step("whole", toks, want=range(75)), ref) < limit
        res = np.frombuffer(s.fab.read(s.lane.residual.data_ptr(), s.lane.residual.numel() * 4), dtype=np.float32)
        res = res.reshape(tuple(s.lane.residual.shape))[:, :75]
        for got, want in zip(res, runs):
            want = want.numpy()
            assert np.sqrt(((got - want) ** 2).mean()) < limit * np.sqrt((want ** 2).mean())
        s.end("whole")
        assert error(run_portions(s, "p", toks, [2, 31, 3, 17, 16, 1]), ref) < limit
        s.end("p")
        assert error(run_portions(s, "d", toks, [2] + [1] * 80), ref) < limit
        s.end("d")
        assert error(run_portions(s, "e", toks, [1]), ref) < limit


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("group", [1, 3, 8])
def test_far_key_through_prompt_and_decoding(dtype, group):
    """One early token's key dominates the scores of every later row, at places around page and key-tile edges: the logits
    far behind it follow it in every schedule, and would not without it.  (The key norm bounds a key, so the query and key
    weights single a direction out: token 7's key points along it, all other keys away from it.)"""
    from monoserve_b200.session import Session
    c = gm.config([gm.parallel((2 * group, 2, 16, 24, 1.5), (1, 1, 8, 8, 2))], 96, 64)
    t = gm.tensors(c, 3)
    t["embed"][:, 0], t["embed"][:, 1], t["embed"][7, 1] = 2.0, -2.0, 8.0
    t["pos"][:, :2] = 0
    q, k = torch.zeros_like(t["l0.mix.left.q"]), 0.02 * t["l0.mix.left.k"].float()
    q[::16, 0] = 4.0   # every head's first column: the same for all tokens
    k[::16, 1] = 4.0   # its sign tells the token apart
    t["l0.mix.left.q"], t["l0.mix.left.k"] = q, k.to(torch.bfloat16)
    t["l0.mix.left.k.norm"] = torch.ones_like(t["l0.mix.left.k.norm"])
    t["l0.mix.left.q.norm"] = torch.ones_like(t["l0.mix.left.q.norm"])
    for place in (0, 15, 16, 127, 128):
        toks = [v if v != 7 else 8 for v in gm.tokens(c, 310, place)]
        without = oracle.model_logits(c, t, toks)
        toks[place] = 7
        ref = oracle.model_logits(c, t, toks)
        limit = limit_of(c, t, toks, ref, dtype)
        assert error(without[-20:], ref[-20:]) > 4 * limit, "the planted key does not show"
        with Session(model_of(c, t, dtype), max_tokens=640, page=16) as s:
            assert error(s.step("a", toks, want=range(310)), ref) < limit
            s.end("a")
            assert error(run_portions(s, "b", toks, [150, 2, 33, 100] + [1] * 40), ref) < limit


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gla", "delta"])
def test_far_write_through_the_memory(kind, dtype):
    """A memory that hardly decays (and, for the delta rule, later keys that do not overwrite it) still shows one strong early
    write hundreds of tokens later, however the tokens were cut; written in the first, a middle and the last token of a step
    of four, and at the edges of a staged chunk."""
    from monoserve_b200.session import Session
    if kind == "gla":
        c = gm.config([gm.gla(2, 16, 24)], 96, 64)
        names = dict(q="l0.mix.q", k="l0.mix.k", v="l0.mix.v")
    else:
        c = gm.config([gm.parallel((1, 1, 8, 8, 1.0), (2, 2, 16, 24, 1))], 96, 64)
        names = dict(q="l0.mix.right.q", k="l0.mix.right.k", v="l0.mix.right.v")
    t = gm.tensors(c, 4)
    t["embed"][:, 0], t["embed"][:, 1], t["embed"][7, 1] = 2.0, 0.0, 8.0
    t["pos"][:, :2] = 0
    if kind == "gla":
        t["l0.mix.a2"].zero_()
        t["l0.mix.a2.b"].fill_(12.0)                  # decay 1 - 4e-7 per token
    else:
        t["l0.mix.right.a2"].zero_()
        t["l0.mix.right.dt_bias"].fill_(-14.0)
        for n in "qkv":
            t[names[n] + ".conv"].fill_(1.0)
        t["l0.mix.left.out"].zero_()                  # the attention beside it does not show
    for n, col in (("q", 0), ("k", 1)):   # a key channel that only token 7 writes, and that every token reads
        w = t[names[n]].float()
        w[::16] = 0
        w[::16, col] = 3.0 if kind == "delta" else 1.0
        if n == "k":
            w[:, 0] = 0
        t[names[n]] = w.to(torch.bfloat16)
    others = torch.arange(32) % 16 != 0
    t[names["q"]][others] = (0.05 * t[names["q"]][others].float()).to(torch.bfloat16)
    for place in (0, 3, 31, 32, 34):
        toks = [v if v != 7 else 8 for v in gm.tokens(c, 300, place)]
        without = oracle.model_logits(c, t, toks)
        toks[place] = 7
        ref = oracle.model_logits(c, t, toks)
        limit = limit_of(c, t, toks, ref, dtype)
        assert error(without[-20:], ref[-20:]) > 4 * limit, "the planted write does not show"
        with Session(model_of(c, t, dtype), max_tokens=640, page=16) as s:
            assert error(s.step("a", toks, want=range(300)), ref) < limit
            s.end("a")
            assert error(run_portions(s, "b", toks, [2, 31, 3, 64, 2, 33, 100] + [1] * 65), ref) < limit


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_portions_run_as_several_passes(dtype):
    """A portion longer than the session's pass, then decode steps whose keys are split over tiles."""
    from monoserve_b200.session import Session
    c = dict(gm.SERVED, max_positions=1200)
    t = gm.tensors(c, 15)
    toks = gm.tokens(c, 1150, 8)
    ref = oracle.model_logits(c, t, toks)
    limit = limit_of(c, t, toks, ref, dtype)
    with Session(model_of(c, t, dtype), max_tokens=1200, page=16, pass_tokens=400) as s:
        assert error(s.step("a", toks[:1130], want=range(1130)), ref[:1130]) < limit
        assert error(run_portions(s, "a", toks[1130:], [1]), ref[1130:]) < limit
        with pytest.raises(ValueError, match="positions"):
            s.step("a", toks[:60])


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_are_used_again(dtype):
    """Requests that come and go over few slots and pages: nothing of an earlier request shows, whatever it left."""
    from monoserve_b200.session import Session
    c = gm.MODELS["mixed"]
    t = gm.tensors(c, 5)
    with Session(model_of(c, t, dtype), max_tokens=96, slots=2, page=8) as s:
        for i, n in enumerate([60, 3, 41, 1, 25]):
            toks = gm.tokens(c, n, 20 + i)
            ref = oracle.model_logits(c, t, toks)
            limit = limit_of(c, t, toks, ref, dtype)
            assert error(run_portions(s, f"r{i}", toks, [[n], [2], [7, 1], [1], [20, 2, 1]][i]), ref) < limit
            if i % 2:   # two requests interleaved, the younger one ends first
                other = gm.tokens(c, 12, 50 + i)
                ref = oracle.model_logits(c, t, other)
                assert error(run_portions(s, "x", other, [5, 1]), ref) < limit_of(c, t, other, ref, dtype)
                s.end("x")
            s.end(f"r{i}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "heads"])
def test_batches_match_each_request_alone(name, dtype):
    """Prompts and portions of unequal requests in one pass, then decode steps of all of them in one program."""
    from monoserve_b200.fabric import Fabric
    from monoserve_b200.layer_list import LayerListCache, LayerListLane
    from tests.test_gpu_model import run_once
    c = gm.MODELS[name]
    t = gm.tensors(c, 7)
    model = model_of(c, t, dtype)
    lengths = [37, 1, 64, 18, 5]
    toks = [gm.tokens(c, n + 6, 30 + i) for i, n in enumerate(lengths)]
    refs = [oracle.model_logits(c, t, v) for v in toks]
    limit = max(limit_of(c, t, v, r, dtype) for v, r in zip(toks, refs))
    fab = Fabric(pool_bytes=256 << 20)
    try:
        kv = LayerListCache(model.cfg, 64, 16, 8)
        lane = LayerListLane(fab, 0, model.cfg, model.weights, kv, max_tokens=160, max_slots=8, bt_stride=8)
        slots = [6, 0, 3, 7, 2]
        for i, slot in enumerate(slots):
            lane.set_pages(slot, [1 + 5 * i + j for j in (3, 0, 4, 1, 2)])
        cuts = [20, 1, 30, 18, 2]   # a first portion of each, then the rest beside it

        def run(h):
            fab.start()
            run_once(fab, h)
            fab.stop()

        run(lane.build_prefill([(s, v[:k], 0) for s, v, k in zip(slots, toks, cuts)], all_logits=True))
        got = lane.logits[:sum(cuts)].cpu()
        assert error(got, torch.cat([r[:k] for r, k in zip(refs, cuts)])) < limit
        rest = [(s, v[k:n], k) for s, v, k, n in zip(slots, toks, cuts, lengths) if n > k]
        run(lane.build_prefill(rest, all_logits=True))
        want = torch.cat([r[k:n] for r, k, n in zip(refs, cuts, lengths) if n > k])
        assert error(lane.logits[:want.shape[0]].cpu(), want) < limit
        for step in range(6):
            for i, slot in enumerate(slots):
                lane.set_request(slot, lengths[i] + step, toks[i][lengths[i] + step])
            order = [(i + step) % 5 for i in range(5)]   # the rows of the batch change places
            run(lane.build_decode([slots[i] for i in order]))
            want = torch.stack([refs[i][lengths[i] + step] for i in order])
            assert error(lane.logits[:5].cpu(), want) < limit
    finally:
        fab.stop()
        fab.close()


def greedy_ok(c, t, prompt, out, slack):
    """Every token is the oracle's arg-max of its own sequence, or within `slack` of the logit range of it."""
    logits = oracle.model_logits(c, t, prompt + out[:-1])
    span = float(logits.max() - logits.min())
    for j, tok in enumerate(out):
        row = logits[len(prompt) - 1 + j]
        assert float(row.max() - row[tok]) <= slack * span, (j, float(row.max() - row[tok]) / span)


@pytest.mark.parametrize("dtype,slack", [("float32", 1e-5), ("bfloat16", 0.02)])
def test_greedy_generation_through_the_serving_loop(dtype, slack):
    """More requests than decode rows, of unequal lengths, through monoserve_b200.generate: continuous batching, slots and
    pages handed on, one long generation."""
    from monoserve_b200.generate import generate
    c = gm.SERVED
    t = gm.tensors(c, 9)
    prompts = [gm.tokens(c, n, 60 + n) for n in (33, 1, 12, 50, 7, 21, 2)]
    results = generate(model_of(c, t, dtype), prompts, max_tokens=40, max_decode=3, token_budget=64)
    for prompt, (out, reason) in zip(prompts, results):
        assert len(out) == 40 and reason == "length"
        greedy_ok(c, t, prompt, out, slack)
    (out, _), = generate(model_of(c, t, dtype), prompts[2:3], max_tokens=400, page=8)
    assert len(out) == 400
    greedy_ok(c, t, prompts[2], out, slack)


def test_trace_replay(tmp_path):
    """bin/trace_run replays steps of a checkpoint folder."""
    c = gm.MODELS["odd"]
    t = gm.tensors(c, 13)
    lm.write(str(tmp_path), c, t)
    toks = gm.tokens(c, 30, 2)
    ref = oracle.model_logits(c, t, toks)
    steps = [dict(step=0, entries=[dict(id="a", tokens=toks[:20], want=[0, 5, 19])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=toks[20:22], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=toks[22:23], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=toks[:7], want=[6])], end=["b"])]
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                           capture_output=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32", "3.f32"]
        for step, rows in ((0, [0, 5, 19]), (2, [22]), (3, [6])):
            got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), c["vocab"])
            assert error(got, ref[rows]) < limit_of(c, t, toks, ref, dtype)

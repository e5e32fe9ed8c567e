"""Layer-list decoders (Sinotar) on a GPU against the plain implementation in oracle/layer_list.py (float64).

Both forms of the programs run the same chain of stages over the same caches and states.  How much a random model
magnifies rounding differs a lot, so a comparison's limit is a few times what rounding-sized noise on every sublayer's
input and output does to the oracle itself: 2^-22 for the 32-bit form, 2^-8 for the bf16 form."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import layer_list as oracle
from tests import layer_list_models as lm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
NOISE = {"float32": 2.0 ** -22, "bfloat16": 2.0 ** -8}
FLOOR = {"float32": 4e-6, "bfloat16": 1.5e-2}


def model_of(c, t, dtype):
    from monoserve_b200 import registry
    from monoserve_b200.layer_list import Weights, read_config
    cfg = read_config(c, dtype)
    return registry.Model(registry._LayerList, cfg, Weights(cfg, t))


def error(got, ref):
    got, ref = torch.as_tensor(np.asarray(got)).double(), torch.as_tensor(ref).double()
    ref_c = ref - ref.mean(-1, keepdim=True)
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1) / ref_c.pow(2).mean()).sqrt().max())


def limit_of(c, t, toks, ref, dtype):
    """Limit of `error` for this model and these tokens."""
    return max(FLOOR[dtype], 4 * error(oracle.model_logits(c, t, toks, jitter=NOISE[dtype]), ref))


def run_portions(session, rid, toks, sizes):
    out, at = [], 0
    while at < len(toks):
        n = min(sizes[len(out) % len(sizes)], len(toks) - at)
        out.append(session.step(rid, toks[at:at + n], want=range(n)))
        at += n
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["scan", "memory", "latent", "ff", "odd", "mixed", "wide", "ones"])
def test_prompt_portions_and_decoding(name, dtype):
    """Whole prompts, portions down to two tokens, and token-by-token decoding give the oracle's logits; the residual
    after every layer run does too (whole prompts)."""
    from monoserve_b200.session import Session
    c = {**lm.ALONE, "odd": lm.ODD, "mixed": lm.MIXED, "wide": lm.WIDE, "ones": lm.ONES}[name]
    t = lm.tensors(c, 11)
    toks = lm.tokens(c, 75, 1)
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_key_through_prompt_and_decoding(dtype):
    """One early token's key is made to dominate the last rows' scores (its latent meets a query direction that all tokens
    share), at places around page edges: the logits far behind it follow it in every schedule, and would not without it."""
    from monoserve_b200.session import Session
    c = lm.config([lm.LATENT], 96, 64, 2)
    t = lm.tensors(c, 3)
    m = c["layers"][0]["mixer"]
    # token 7 carries direction u in the embedding; W_q maps a constant column of every token onto its key
    t["embed"][:, 0] = 6.0
    t["embed"][:, 1] = 0.0
    t["embed"][7, 1] = 24.0
    q = torch.zeros_like(t["l0.mix.q"])
    dkv, uk = t["l0.mix.dkv"].clone(), t["l0.mix.uk"].clone()
    dkv[0, :] = 0
    dkv[0, 1] = 3.0
    for h in range(m["heads"]):
        q[h * (m["dim"] + m["rot_dim"]), 0] = 4.0
        uk[h * m["dim"], :] = 0
        uk[h * m["dim"], 0] = 2.0
    t["l0.mix.q"], t["l0.mix.dkv"], t["l0.mix.uk"] = q, dkv, uk
    for place in (0, 15, 16, 31):
        toks = [v if v != 7 else 8 for v in lm.tokens(c, 210, place)]
        without = oracle.model_logits(c, t, toks)
        toks[place] = 7
        ref = oracle.model_logits(c, t, toks)
        limit = limit_of(c, t, toks, ref, dtype)
        assert error(without[-20:], ref[-20:]) > 4 * limit, "the planted key does not show"
        with Session(model_of(c, t, dtype), max_tokens=512, page=16) as s:
            assert error(s.step("a", toks, want=range(210)), ref) < limit
            s.end("a")
            assert error(run_portions(s, "b", toks, [150, 2, 33] + [1] * 40), ref) < limit


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_run_as_several_passes(dtype):
    """A portion longer than the session's pass: several programs, whole-prompt attention for the first and the cached
    latents for the rest, several key tiles; then decode steps whose keys are split over tiles."""
    from monoserve_b200.session import Session
    c = lm.SERVED
    t = lm.tensors(c, 15)
    toks = lm.tokens(c, 420, 8)
    ref = oracle.model_logits(c, t, toks)
    limit = limit_of(c, t, toks, ref, dtype)
    with Session(model_of(c, t, dtype), max_tokens=512, page=16, pass_tokens=160) as s:
        assert error(s.step("a", toks[:400], want=range(400)), ref[:400]) < limit
        assert error(run_portions(s, "a", toks[400:], [1]), ref[400:]) < limit


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_are_used_again(dtype):
    """Requests that come and go over few slots and pages: nothing of an earlier request shows, whatever it left."""
    from monoserve_b200.session import Session
    c = lm.MIXED
    t = lm.tensors(c, 5)
    with Session(model_of(c, t, dtype), max_tokens=96, slots=2, page=8) as s:
        for i, n in enumerate([60, 3, 41, 1, 25]):
            toks = lm.tokens(c, n, 20 + i)
            ref = oracle.model_logits(c, t, toks)
            limit = limit_of(c, t, toks, ref, dtype)
            assert error(run_portions(s, f"r{i}", toks, [[n], [2], [7, 1], [1], [20, 2, 1]][i]), ref) < limit
            if i % 2:   # two requests interleaved, the younger one ends first
                other = lm.tokens(c, 12, 50 + i)
                ref = oracle.model_logits(c, t, other)
                assert error(run_portions(s, "x", other, [5, 1]), ref) < limit_of(c, t, other, ref, dtype)
                s.end("x")
            s.end(f"r{i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_batches_match_each_request_alone(name, dtype):
    """Prompts and portions of unequal requests in one pass, then decode steps of all of them in one program."""
    from monoserve_b200.fabric import Fabric
    from monoserve_b200.layer_list import LayerListCache, LayerListLane
    from tests.test_gpu_model import run_once
    c = lm.MIXED if name == "mixed" else lm.ODD
    t = lm.tensors(c, 7)
    model = model_of(c, t, dtype)
    lengths = [37, 1, 64, 18, 5]
    toks = [lm.tokens(c, n + 6, 30 + i) for i, n in enumerate(lengths)]
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
    c = lm.SERVED
    t = lm.tensors(c, 9)
    prompts = [lm.tokens(c, n, 60 + n) for n in (33, 1, 12, 50, 7, 21, 2)]
    results = generate(model_of(c, t, dtype), prompts, max_tokens=40, max_decode=3, token_budget=64)
    for prompt, (out, reason) in zip(prompts, results):
        assert len(out) == 40 and reason == "length"
        greedy_ok(c, t, prompt, out, slack)
    (out, _), = generate(model_of(c, t, dtype), prompts[2:3], max_tokens=400, page=8)
    assert len(out) == 400
    greedy_ok(c, t, prompts[2], out, slack)


def test_command_lines(tmp_path):
    """bin/trace_run replays steps of a checkpoint folder; monoserve_b200.generate continues a prompt of it."""
    c = lm.ODD
    t = lm.tensors(c, 13)
    lm.write(str(tmp_path), c, t)
    toks = lm.tokens(c, 30, 2)
    ref = oracle.model_logits(c, t, toks)
    limit = {dtype: limit_of(c, t, toks, ref, dtype) for dtype in NOISE}
    steps = [dict(step=0, entries=[dict(id="a", tokens=toks[:20], want=[0, 5, 19])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=toks[20:22], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=toks[22:23], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=toks[:7], want=[6])], end=["b"])]
    for dtype in ("float32", "bfloat16"):
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
            assert error(got, ref[rows]) < limit[dtype]
    r = subprocess.run([sys.executable, "-m", "monoserve_b200.generate", "--model", str(tmp_path), "--prompt",
                        ",".join(map(str, toks[:9])), "--max-tokens", "5", "--dtype", "float32"], text=True, cwd=ROOT,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    out = json.loads(r.stdout.splitlines()[-1])["tokens"]
    assert len(out) == 5
    greedy_ok(c, t, toks[:9], out, 1e-5)

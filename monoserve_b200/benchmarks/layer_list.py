"""Layer-list decoders beside the closest models of the library: prefill and decode throughput at layer sizes of real
models, random weights, three layers with their feed-forward.  --design Sinotar (matrix memory, selective scan, latent
attention; 4 residual streams) or Teganex (gated linear attention of two shapes around an attention / delta rule layer), and
always `dense`: the dense-layer form of the GLM-style decoder (grouped-query attention and a gated feed-forward) at equal
width, depth and feed-forward.  With Teganex the Sinotar layers are run as well: they have the like recurrence stages.

    python -m monoserve_b200.benchmarks.layer_list [--design Sinotar] [--sizes 2048,4096] [--steps 20] [--only ...] [--stages]
                                                  [--serial]

Timed by the fabric's iteration timer (device clock) over repeating programs on all SMs: `prefill` = 4 prompts of 1024
tokens per iteration, `decode` = one token of 32 sequences with contexts around 4096 per iteration.  The weights of a
step (more than 250 MB) exceed L2.  Every stage's mean span comes with its roofline time: the larger of its algorithmic
bytes over the measured copy bandwidth and its products' FLOPs over the measured bf16 GEMM rate (MEASURED_PEAKS.json),
and `frac` = roofline time / span.  One JSON line; --stages prints the tables to stderr.  Stages that do not depend on one
another share the SMs, and their spans include one another's work; --serial chains the stages of the layer-list decoders, for
the spans of each alone.
"""
import argparse
import json
import os
import sys
import types

import numpy as np
import torch

PEAKS = dict(hbm_gbs=6650.0, bf16_tflops=1590.0)
_path = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "..", "MEASURED_PEAKS.json")
if os.path.exists(_path):
    with open(_path) as _f:
        PEAKS.update({k: v for k, v in json.load(_f).items() if k in PEAKS})

PROMPTS, PROMPT_LEN, DECODE_ROWS, CONTEXT, PAGE, VOCAB = 4, 1024, 32, 4096, 16, 32768


def teganex_config(W):
    """A layer of many small memories, one with attention beside the delta rule, one of few large memories (the size of the
    matrix memory's)."""
    from monoserve_b200.layer_list import read_config
    mixers = [("gla", dict(heads=W // 128, dim=64, vdim=128, tau=16.0)),
              ("parallel", dict(left=dict(heads=W // 128, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5),
                                right=dict(heads=W // 128, kv_heads=W // 256, dim=128, vdim=128, conv=4))),
              ("gla", dict(heads=W // 512, dim=256, vdim=512, tau=16.0))]
    return read_config(dict(architecture="Teganex", layers=[dict(type=k, mixer=m, mlp=dict(kind="dense", ff=3 * W)) for k, m in mixers],
                            width=W, vocab=VOCAB, norm=dict(eps=1e-5), embedding=dict(scale=1.0), logit_scale=1.0,
                            max_positions=CONTEXT * 2))


def teganex_tensors(cfg):
    """Random tensors, made on the device."""
    W, t = cfg.hidden, {}
    g = torch.Generator(device="cuda").manual_seed(0)
    r = lambda *shape, scale=1.0: (torch.randn(*shape, generator=g, device="cuda") * scale).to(torch.bfloat16)  # noqa: E731
    lin = lambda o, i: r(o, i, scale=i ** -0.5)  # noqa: E731
    one = lambda n: 1 + r(n, scale=0.1)  # noqa: E731
    t.update({"embed": r(cfg.vocab, W), "pos": r(cfg.max_positions, W, scale=0.1), "head": lin(cfg.vocab, W), "final.norm": one(W)})
    for i, layer in enumerate(cfg.layers):
        m, p, x = layer.m, f"l{i}.", f"l{i}.mix."
        for n in ("norm1", "norm1b", "norm2", "norm2b"):
            t[p + n] = one(W)
        if layer.kind == "gla":
            H, d, e = m.heads, m.dim, m.vdim
            for n, o in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e), ("a1", 16)):
                t[x + n] = lin(o, W)
            t[x + "a2"], t[x + "a2.b"], t[x + "norm"], t[x + "o"] = lin(H * d, 16), r(H * d) + 2, one(e), lin(W, H * e)
        else:
            a = m.left
            for n, o in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim), ("g", a.heads)):
                t[f"{x}left.{n}"] = lin(o, W)
            t[x + "left.q.norm"], t[x + "left.k.norm"], t[x + "left.o"] = one(a.dim), one(a.dim), lin(W, a.heads * a.vdim)
            a = m.right
            for n, o in (("q", a.kv_heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.heads * a.vdim)):
                t[f"{x}right.{n}"], t[f"{x}right.{n}.conv"] = lin(o, W), r(o, a.conv, scale=0.5)
            for n, o in (("b", a.heads), ("a1", a.dim), ("g1", a.vdim)):
                t[f"{x}right.{n}"] = lin(o, W)
            t[x + "right.a2"], t[x + "right.g2"] = lin(a.heads * a.dim, a.dim), lin(a.heads * a.vdim, a.vdim)
            t[x + "right.A_log"], t[x + "right.dt_bias"] = r(a.heads), r(a.heads * a.dim) - 3
            t[x + "right.norm"], t[x + "right.o"] = one(a.vdim), lin(W, a.heads * a.vdim)
            t[x + "left.out"], t[x + "right.out"] = one(W), one(W)
        t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = lin(layer.ff, W), lin(layer.ff, W), lin(W, layer.ff)
    return t


def new_config(W):
    from monoserve_b200.layer_list import read_config
    mixers = [("mlstm", dict(heads=W // 512, dim=256, vdim=512, gate_cap=15.0)),
              ("mamba1", dict(inner=2 * W, state=16, dt_rank=W // 16, conv=4)),
              ("latent_attention", dict(heads=W // 128, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5,
                                        rot=dict(base=1e4, dims=64)))]
    return read_config(dict(layers=[dict(type=k, mixer=m, mlp=dict(kind="dense", ff=3 * W)) for k, m in mixers], width=W,
                            vocab=VOCAB, streams=4, norm=dict(eps=1e-5)))


def new_tensors(cfg):
    """Random tensors, made on the device."""
    W, s, t = cfg.hidden, cfg.streams, {}
    g = torch.Generator(device="cuda").manual_seed(0)
    r = lambda *shape, scale=1.0: (torch.randn(*shape, generator=g, device="cuda") * scale).to(torch.bfloat16)  # noqa: E731
    lin = lambda o, i: r(o, i, scale=i ** -0.5)  # noqa: E731
    t["embed"], t["head"], t["final.norm"] = r(cfg.vocab, W), lin(cfg.vocab, W), r(W, scale=0.1)
    for i, layer in enumerate(cfg.layers):
        m, p = layer.m, f"l{i}."
        for q in (1, 2):
            t[f"{p}norm{q}"], t[f"{p}hc{q}.in"] = r(W, scale=0.1), torch.full((s,), 1.0 / s)
            t[f"{p}hc{q}.out"], t[f"{p}hc{q}.mix"] = torch.full((s,), 0.5), torch.eye(s)
        x = p + "mix."
        if layer.kind == "mamba1":
            C = m.inner
            t[x + "in"], t[x + "conv"], t[x + "conv.b"] = lin(2 * C, W), r(C, m.conv, scale=0.5), r(C, scale=0.1)
            t[x + "x"], t[x + "dt"], t[x + "dt.b"] = lin(m.dt_rank + 2 * m.state, C), lin(C, m.dt_rank), r(C) - 3
            t[x + "A_log"], t[x + "D"], t[x + "o"] = r(C, m.state, scale=0.5), r(C), lin(W, C)
        elif layer.kind == "mlstm":
            H, d, e = m.heads, m.dim, m.vdim
            for n, o in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e), ("i", H), ("f", H)):
                t[x + n] = lin(o, W)
            t[x + "i.b"], t[x + "f.b"], t[x + "norm"], t[x + "o"] = r(H), r(H) + 3, 1 + r(H * e, scale=0.1), lin(W, H * e)
        else:
            H, d, rr, e, k = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
            t[x + "q"], t[x + "dkv"], t[x + "dkv.norm"] = lin(H * (d + rr), W), lin(k + rr, W), 1 + r(k, scale=0.1)
            t[x + "uk"], t[x + "uv"], t[x + "o"] = lin(H * d, k), lin(H * e, k), lin(W, H * e)
        t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = lin(layer.ff, W), lin(layer.ff, W), lin(W, layer.ff)
    return t


def dense_config(W):
    return types.SimpleNamespace(hidden=W, intermediate=64, num_experts=8, top_k=1, num_layers=3, dense_layers=3,
                                 dense_intermediate=3 * W, shared_intermediate=0, num_heads=W // 128, num_kv_heads=8, head_dim=128,
                                 vocab=VOCAB, rope_theta=1e6, rms_eps=1e-6, rotary_dim=128)


def dense_weights(cfg):
    from monoserve_b200.model import ModelWeights
    W, L, D, F = cfg.hidden, cfg.num_layers, cfg.num_heads * 128, cfg.dense_intermediate
    g = torch.Generator(device="cuda").manual_seed(0)
    r = lambda *shape: (torch.randn(*shape, generator=g, device="cuda") * shape[-1] ** -0.5).to(torch.bfloat16)  # noqa: E731
    one = lambda n: torch.ones(n, dtype=torch.bfloat16, device="cuda")  # noqa: E731
    w = types.SimpleNamespace(embed=r(cfg.vocab, W), lm_head=r(cfg.vocab, W), final_norm=one(W))
    w.in_norm, w.post_norm = [one(W) for _ in range(L)], [one(W) for _ in range(L)]
    w.q_norm, w.k_norm = [one(128) for _ in range(L)], [one(128) for _ in range(L)]
    w.qkv, w.o = [r(D + 2 * cfg.num_kv_heads * 128, W) for _ in range(L)], [r(W, D) for _ in range(L)]
    w.mlp_w13, w.mlp_w2 = [r(2 * F, W) for _ in range(L)], [r(W, F) for _ in range(L)]
    w.router = w.host_w13 = w.host_w2 = [None] * L
    return ModelWeights(cfg, w)


# ------------------------------------------------------------------------------------------ rooflines
def seconds(nbytes, flops=0.0):
    return max(nbytes / (PEAKS["hbm_gbs"] * 1e9), flops / (PEAKS["bf16_tflops"] * 1e12))


def gemm(T, n, k, out_bytes):
    return seconds(2 * (n * k + T * k) + out_bytes * T * n, 2.0 * T * n * k)


def new_roofline(cfg, T, R, pairs, keys):
    """{stage: roofline seconds}; T rows, R requests, pairs = (query, key) pairs, keys = cached keys read."""
    W, s, f = cfg.hidden, cfg.streams, cfg.layers[0].ff
    st = {"streams": seconds(T * W * (8.0 * s + 4 + 2)), "streams_ff": seconds(T * W * (8.0 * s + 4 + 2)),
          "final": seconds(T * W * (8.0 * s + 4)), "ff_in": gemm(T, 2 * f, W, 1), "ff_out": gemm(T, W, f, 4),
          "head": gemm(R, cfg.vocab, W, 4), "sample": seconds(4.0 * R * cfg.vocab)}
    for layer in cfg.layers:
        m = layer.m
        if layer.kind == "mamba1":
            C, n, r = m.inner, m.state, m.dt_rank
            st.update(scan_in=gemm(T, 2 * C, W, 2), conv=seconds(4.0 * T * C), scan_x=gemm(T, r + 2 * n, C, 4),
                      scan_sum=seconds(T * (8.0 * (r + 2 * n) + 2 * r)), scan_dt=gemm(T, C, r, 4),
                      scan=seconds(T * (C * 10.0 + 8 * n) + 8.0 * R * C * n), scan_o=gemm(T, W, C, 4))
        elif layer.kind == "mlstm":
            H, d, e = m.heads, m.dim, m.vdim
            st.update(memory_in=gemm(T, 2 * H * (d + e), W, 2), memory_gates=seconds(4.0 * T * W),
                      memory=seconds(T * H * (4.0 * d + 6 * e) + 8.0 * R * H * d * e, 6.0 * T * H * d * e),
                      head_norm=seconds(8.0 * T * H * e), memory_o=gemm(T, W, H * e, 4))
        else:
            H, d, r, e, k = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
            # attention: the cheaper of the two forms' FLOPs per pair, and the latents read once per request
            per_pair = 2.0 * H * (d + r + e) if T > R else 2.0 * H * (2 * k + r)
            st.update(latent_in=gemm(T, H * (d + r) + k + r, W, 4), latent_kv=seconds(T * (H * (d + r) + k + r) * 6.0),
                      latent_q=seconds(2.0 * H * k * d + T * H * 2.0 * (d + k), 2.0 * T * H * k * d),
                      latent_attn=seconds(2.0 * keys * (k + r), pairs * per_pair),
                      latent_merge=seconds(2.0 * T * H * k),
                      latent_v=seconds(2.0 * H * k * e + T * H * 2.0 * (e + k), 2.0 * T * H * k * e), latent_o=gemm(T, W, H * e, 4))
    return st


def teganex_roofline(cfg, T, R, pairs, keys):
    """As new_roofline; stages of the two kinds of gla layers are told apart by their layer."""
    W, f = cfg.hidden, cfg.layers[0].ff
    row = lambda ys: seconds(T * W * (8.0 + 4 * ys + 2))  # noqa: E731
    st = {"residual": row(1), "residual_ff": row(1), "final": seconds(T * W * 12.0), "residual_ff.1": row(2),
          "ff_in": gemm(T, 2 * f, W, 1), "ff_out": gemm(T, W, f, 4), "head": gemm(R, cfg.vocab, W, 4), "sample": seconds(4.0 * R * cfg.vocab)}
    # a memory: its inputs and outputs, its state read and written once, six operations per token and state element
    memory = lambda H, G, d, e: seconds(T * (4.0 * G * d + 4 * H * d + 6 * H * e) + 8.0 * R * H * d * e, 6.0 * T * H * d * e)  # noqa: E731
    for i, layer in enumerate(cfg.layers):
        m = layer.m
        if layer.kind == "gla":
            H, d, e = m.heads, m.dim, m.vdim
            st.update({f"gla_in.{i}": gemm(T, 2 * H * (d + e), W, 2), f"gla_decay.{i}": seconds(T * (4.0 * H * d + 32)),
                       f"gla.{i}": memory(H, H, d, e), f"gla_norm.{i}": seconds(8.0 * T * H * e), f"gla_o.{i}": gemm(T, W, H * e, 4)})
        else:
            a, b = m.left, m.right
            H, G, d, e = a.heads, a.kv_heads, a.dim, a.vdim
            C = 2 * b.kv_heads * b.dim + b.heads * b.vdim
            n = H * d + G * (d + e) + H + C + b.heads + b.dim + b.vdim
            st.update(parallel_in=gemm(T, n, W, 2), qkv=seconds(4.0 * T * (H * d + G * (d + e))),
                      attn=seconds(2.0 * keys * G * (d + e), 2.0 * pairs * H * (d + e)), head_gate=seconds(4.0 * T * H * e),
                      attn_o=gemm(T, W, H * e, 4), delta_conv=seconds(4.0 * T * C), delta_decay=seconds(T * (4.0 * b.heads * b.dim + 2 * b.dim)),
                      delta_gate=gemm(T, b.heads * b.vdim, b.vdim, 2), delta=memory(b.heads, b.kv_heads, b.dim, b.vdim),
                      delta_norm=seconds(8.0 * T * b.heads * b.vdim), delta_o=gemm(T, W, b.heads * b.vdim, 4))
    return st


def dense_roofline(cfg, T, R, pairs, keys):
    W, f, hq, hkv = cfg.hidden, cfg.dense_intermediate, cfg.num_heads, cfg.num_kv_heads
    q = (hq + 2 * hkv) * 128
    return {"embed": seconds(6.0 * T * W), "qkv": gemm(T, q, W, 2), "rope": seconds(4.0 * T * q),
            "attn": seconds(keys * hkv * 512.0, pairs * hq * 512.0), "o": gemm(T, W, hq * 128, 4), "norm": seconds(4.0 * T * W),
            "in_norm": seconds(4.0 * T * W), "final_norm": seconds(4.0 * T * W), "mlp_w13": gemm(T, 2 * f, W, 1),
            "mlp_w2": gemm(T, W, f, 4), "lm_head": gemm(R, cfg.vocab, W, 4), "sample": seconds(4.0 * R * cfg.vocab)}


# ------------------------------------------------------------------------------------------ runs
def timed(fab, lane, handle, tokens, steps, roofline, show):
    from monoserve_b200.fabric.trace import StageTrace, spans
    tr = StageTrace(capacity=1 << 19)
    torch.cuda.synchronize()

    fab.start()
    fab.publish(map=[0] * fab.num_workers, caps=[4], order=[0], programs=[handle])
    ends = fab.iteration_times(0, 0, 3 + steps, timeout=120)
    ms = np.diff(np.array(ends[2:], dtype=np.float64)) * 1e-6
    tr.start(fab)   # the stage spans come from iterations of their own
    at = fab.iterations(0)
    fab.iteration_times(0, at, 2 + steps, timeout=120)
    records = tr.stop(fab)
    error = fab.progress()["error"]
    fab.stop()
    if error:
        raise RuntimeError(f"device error {error:#x}: {fab.wait_notes()}")
    us = {}
    for name, layer, _, t0, t1 in spans(records, lane.labels, 0):
        one = f"{name}.{layer}"   # stages that differ from layer to layer
        us.setdefault(one if one in roofline or name.startswith("gla") else name, []).append((t1 - t0) / 1e3)
    stages = {}
    for name, v in us.items():
        mean = float(np.median(v))
        r = roofline.get(name)
        stages[name] = dict(us=round(mean, 2), per_iteration=round(len(v) / max(1, steps), 1),
                            roofline_us=None if r is None else round(r * 1e6, 2), frac=None if r is None else round(r * 1e6 / mean, 3))
    if show:
        for name, v in sorted(stages.items(), key=lambda kv: -kv[1]["us"]):
            print(f"{name:14s} {v['us']:9.1f} us  roofline {v['roofline_us']}  frac {v['frac']}", file=sys.stderr)
        print(file=sys.stderr)
    return dict(ms=round(float(np.median(ms)), 4), tokens_per_s=round(tokens / float(np.median(ms)) * 1e3, 1), stages=stages)


def serial_program():
    from monoserve_b200.fabric import Program

    class Serial(Program):
        """Every stage waits for the one added before it."""
        last = None

        def stage(self, *args, **kwargs):
            s = super().stage(*args, **kwargs)
            if self.last is not None:
                self.after(self.last, s)
            self.last = s
            return s
    return Serial


def fabric():
    from monoserve_b200.fabric import Fabric
    fab = Fabric(pool_bytes=512 << 20)
    fab.set_max_run(300)
    return fab


def measure(kind, W, steps, show, serial=False):
    from monoserve_b200.layer_list import LayerListCache, LayerListLane, Weights
    from monoserve_b200.model import KVCache, ModelLane
    rng = np.random.default_rng(0)
    listed = kind != "dense"
    if listed:
        make_config, make_tensors, roofline = {"Sinotar": (new_config, new_tensors, new_roofline),
                                               "Teganex": (teganex_config, teganex_tensors, teganex_roofline)}[kind]
        cfg = make_config(W)
        weights = Weights(cfg, make_tensors(cfg))
    else:
        cfg, roofline = dense_config(W), dense_roofline
        weights = dense_weights(cfg)
    ctx = rng.integers(CONTEXT // 2, CONTEXT * 3 // 2, size=DECODE_ROWS)
    grow = 4 * steps + 64
    dec_pages = [-(-(int(n) + grow) // PAGE) for n in ctx]
    pre_pages = -(-PROMPT_LEN // PAGE)
    n_pages = 1 + sum(dec_pages) + PROMPTS * pre_pages
    kv = LayerListCache(cfg, n_pages, PAGE, DECODE_ROWS) if listed else KVCache(cfg, n_pages, PAGE)
    if listed:
        for run in kv.runs:
            for t in run.values():
                t.normal_(0, 0.5)
    else:
        for t in kv.k + kv.v:
            t.normal_(0, 1)
    make = LayerListLane if listed else ModelLane
    programs = dict(program=serial_program()) if serial and listed else {}
    out = {}
    fab = fabric()   # one per program: a stopped lane keeps the program it was running
    try:
        T = PROMPTS * PROMPT_LEN
        stride = max(dec_pages)
        perm = rng.permutation(n_pages - 1) + 1
        lane = make(fab, 0, cfg, weights, kv, max_tokens=T, max_slots=DECODE_ROWS, bt_stride=stride, logit_rows=DECODE_ROWS)
        vars(lane).update(programs)
        at, batch = 0, []
        for s in range(PROMPTS):
            lane.set_pages(s, perm[at:at + pre_pages].tolist())
            at += pre_pages
            batch.append((s, rng.integers(0, cfg.vocab, size=PROMPT_LEN).tolist(), 0))
        pairs, keys = PROMPTS * PROMPT_LEN * (PROMPT_LEN + 1) / 2, T
        roof = roofline(cfg, T, PROMPTS, pairs, keys)
        h = lane.build_prefill(batch, iterations=0)
        out["prefill"] = timed(fab, lane, h, T, steps, roof, show)
        fab.close()
        del lane
        fab = fabric()
        lane = make(fab, 0, cfg, weights, kv, max_tokens=DECODE_ROWS, max_slots=DECODE_ROWS, bt_stride=stride, logit_rows=DECODE_ROWS)
        vars(lane).update(programs)
        for s, n in enumerate(dec_pages):
            lane.set_pages(s, perm[at:at + n].tolist())
            at += n
            lane.set_request(s, seq_len=int(ctx[s]), last_token=int(rng.integers(0, cfg.vocab)))
        keys = float(ctx.sum())
        roof = roofline(cfg, DECODE_ROWS, DECODE_ROWS, keys, keys)
        h = lane.build_decode(list(range(DECODE_ROWS)), iterations=0)
        out["decode"] = timed(fab, lane, h, DECODE_ROWS, steps, roof, show)
    finally:
        fab.stop()
        fab.close()
    return out


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="2048,4096", help="model widths")
    ap.add_argument("--steps", type=int, default=20)
    ap.add_argument("--design", choices=["Sinotar", "Teganex"], default="Sinotar")
    ap.add_argument("--only", choices=["Sinotar", "Teganex", "dense"])
    ap.add_argument("--stages", action="store_true")
    ap.add_argument("--serial", action="store_true")
    args = ap.parse_args(argv)
    what = {"Sinotar": "matrix memory, selective scan, latent attention; 4 residual streams",
            "Teganex": "gated linear attention, attention beside a gated delta rule, gated linear attention of few large heads"}[args.design]
    line = {"workload": f"layer-list decoder {args.design} ({what}) beside the "
                        f"dense-layer decoder, 3 layers each, ff 3 x width; prefill {PROMPTS} x {PROMPT_LEN}, decode {DECODE_ROWS} "
                        f"sequences at contexts {CONTEXT // 2}..{CONTEXT * 3 // 2}", "dtype": "bf16", "data": "synthetic",
            "l2": "the weights of a step exceed L2", "peaks": PEAKS, "sizes": {}}
    kinds = ("Sinotar", "dense") if args.design == "Sinotar" else ("Teganex", "Sinotar", "dense")
    for W in [int(v) for v in args.sizes.split(",")]:
        line["sizes"][W] = {}
        for kind in (args.only,) if args.only else kinds:
            if args.stages:
                print(f"== width {W}, {kind}", file=sys.stderr)
            line["sizes"][W][kind] = measure(kind, W, args.steps, args.stages, args.serial)
            torch.cuda.empty_cache()
    print(json.dumps(line), flush=True)


if __name__ == "__main__":
    main()

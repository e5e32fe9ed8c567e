"""Small random layer-list models for the tests: configurations, tensors, and their checkpoint folders."""
import json
import os

import torch


def scan(inner, state, dt_rank, conv):
    return "mamba1", dict(inner=inner, state=state, dt_rank=dt_rank, conv=conv)


def memory(heads, dim, vdim, cap):
    return "mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def latent(heads, dim, rot, vdim, rank, base, scale):
    return "latent_attention", dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, scale=scale,
                                    rot=dict(base=base, dims=rot))


def config(layers, width, vocab, streams, ff=None, loop=None, eps=1e-5):
    """layers: mixers, or (mixer, ff) pairs; ff: the feed-forward width of layers that name none (None: no feed-forward)."""
    out = []
    for entry in layers:
        (kind, mixer), f = entry if isinstance(entry[0], tuple) else (entry, ff)
        out.append(dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=f) if f else None))
    c = dict(architecture="Sinotar", layers=out, width=width, vocab=vocab, streams=streams, norm=dict(eps=eps))
    if loop:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


def tensors(c, seed):
    """Random tensors in bf16: outputs of every sublayer of order one, gates and decays spread over short and long memory."""
    g = torch.Generator().manual_seed(seed)
    W, V, s = c["width"], c["vocab"], c["streams"]
    t = {}

    def put(name, *shape, scale=1.0, at=0.0):
        t[name] = (at + scale * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    def lin(name, out, inp, gain=1.0):
        put(name, out, inp, scale=gain * inp ** -0.5)

    put("embed", V, W)
    lin("head", V, W)
    put("final.norm", W, scale=0.2)
    for i, layer in enumerate(c["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer["mlp"] else (1,):
            put(f"{p}norm{q}", W, scale=0.2)
            put(f"{p}hc{q}.in", s, scale=0.5 / s, at=1.0 / s)
            put(f"{p}hc{q}.out", s, scale=0.3, at=0.5)
            t[f"{p}hc{q}.mix"] = (0.8 * torch.eye(s) + 0.3 / s * torch.randn(s, s, generator=g)).to(torch.bfloat16)
        x = p + "mix."
        if layer["type"] == "mamba1":
            C, n, r = m["inner"], m["state"], m["dt_rank"]
            lin(x + "in", 2 * C, W)
            put(x + "conv", C, m["conv"], scale=0.6)
            put(x + "conv.b", C, scale=0.3)
            lin(x + "x", r + 2 * n, C)
            lin(x + "dt", C, r)
            t[x + "dt.b"] = (-4 + 4 * torch.rand(C, generator=g)).to(torch.bfloat16)
            t[x + "A_log"] = (torch.rand(C, n, generator=g) * 4 - 3).to(torch.bfloat16)
            put(x + "D", C)
            lin(x + "o", W, C)
        elif layer["type"] == "mlstm":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            for name, n in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e)):
                lin(x + name, n, W)
            # queries near the keys: the head norm after the memory magnifies a read-out that nearly cancels
            t[x + "q"] = (2 * t[x + "k"].float() + t[x + "q"].float()).to(torch.bfloat16)
            lin(x + "i", H, W, 2.0)
            lin(x + "f", H, W, 2.0)
            put(x + "i.b", H)
            put(x + "f.b", H, scale=1.5, at=3.0)
            put(x + "norm", H * e, scale=0.2, at=1.0)
            lin(x + "o", W, H * e)
        else:
            H, d, r, e, k = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            lin(x + "q", H * (d + r), W, 2.0)
            lin(x + "dkv", k + r, W, 1.5)
            put(x + "dkv.norm", k, scale=0.3, at=1.0)
            lin(x + "uk", H * d, k)
            lin(x + "uv", H * e, k)
            lin(x + "o", W, H * e)
        if layer["mlp"]:
            f = layer["mlp"]["ff"]
            lin(p + "mlp.gate", f, W)
            lin(p + "mlp.up", f, W)
            lin(p + "mlp.down", W, f)
    return t


def write(folder, c, t):
    from monoserve_b200.checkpoint import write_safetensors
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(c, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), t)


def tokens(c, n, seed):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


SCAN = scan(inner=72, state=16, dt_rank=8, conv=4)
MEMORY = memory(heads=3, dim=24, vdim=40, cap=8.0)
LATENT = latent(heads=5, dim=24, rot=8, vdim=40, rank=72, base=3000.0, scale=0.2)
# every mechanism with sizes that are no multiple of anything the kernels like
ODD = config([scan(inner=75, state=5, dt_rank=7, conv=3), (latent(heads=3, dim=19, rot=6, vdim=21, rank=45, base=700.0, scale=0.31), 53),
              (memory(heads=2, dim=18, vdim=35, cap=5.0), None), scan(inner=33, state=33, dt_rank=1, conv=1)],
             width=90, vocab=203, streams=5, ff=41, loop=(1, 3, 3), eps=3e-4)
MIXED = config([MEMORY, LATENT, SCAN, LATENT], width=112, vocab=160, streams=2, ff=96, loop=(1, 3, 2))
WIDE = config([(scan(inner=520, state=64, dt_rank=40, conv=5), None), latent(heads=17, dim=64, rot=32, vdim=96, rank=320, base=1e4, scale=0.1),
               memory(heads=1, dim=300, vdim=65, cap=15.0), (memory(heads=4, dim=130, vdim=31, cap=15.0), None)],
              width=1100, vocab=333, streams=4, ff=700)
SERVED = config([LATENT, SCAN, MEMORY], width=112, vocab=160, streams=2, ff=64)   # magnifies rounding little
ONES = config([scan(inner=1, state=1, dt_rank=1, conv=2), latent(heads=1, dim=1, rot=2, vdim=1, rank=1, base=10.0, scale=1.0),
               memory(heads=1, dim=1, vdim=2, cap=1.0)], width=16, vocab=16, streams=1, ff=1)
ALONE = {"scan": config([SCAN], 96, 128, 3), "memory": config([MEMORY], 96, 128, 3), "latent": config([LATENT], 96, 128, 3),
         "ff": config([(scan(inner=8, state=1, dt_rank=1, conv=1), 80)], 96, 128, 4)}


def copy_of(c):
    return json.loads(json.dumps(c))

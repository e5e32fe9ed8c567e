"""Small random Teganex models for the tests: configurations and tensors."""
import torch


def gla(heads, dim, vdim, tau=16.0):
    return "gla", dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def parallel(left, right):
    """left: (heads, kv_heads, dim, vdim, scale); right: (heads, kv_heads, dim, vdim, conv)."""
    return "parallel", dict(left=dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left)),
                            right=dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right)))


def config(layers, width, vocab, ff=None, eps=2e-5, embed=2.5, logits=1.5, positions=512):
    """layers: mixers, or (mixer, ff) pairs; ff: the feed-forward width of layers that name none (None: no feed-forward)."""
    out = []
    for entry in layers:
        (kind, mixer), f = entry if isinstance(entry[0], tuple) else (entry, ff)
        out.append(dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=f) if f else None))
    return dict(architecture="Teganex", layers=out, width=width, vocab=vocab, norm=dict(eps=eps), embedding=dict(scale=embed),
                logit_scale=logits, max_positions=positions)


def tensors(c, seed, rank=None):
    """Random tensors in bf16: outputs of every sublayer of order one, decays spread over short and long memory.  rank: of the
    decay and gate projections (a number per projection otherwise)."""
    g = torch.Generator().manual_seed(seed)
    W, V = c["width"], c["vocab"]
    t = {}

    def put(name, *shape, scale=1.0, at=0.0):
        t[name] = (at + scale * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    def lin(name, out, inp, gain=1.0):
        put(name, out, inp, scale=gain * inp ** -0.5)

    def uniform(name, n, lo, hi):
        t[name] = (lo + (hi - lo) * torch.rand(n, generator=g)).to(torch.bfloat16)

    put("embed", V, W, scale=0.4)
    put("pos", c["max_positions"], W, scale=0.4)
    lin("head", V, W)
    put("final.norm", W, scale=0.2, at=1.0)
    for i, layer in enumerate(c["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer["mlp"] else (1,):
            put(f"{p}norm{q}", W, scale=0.2, at=1.0)
            put(f"{p}norm{q}b", W, scale=0.2, at=0.7)
        x = p + "mix."
        if layer["type"] == "gla":
            H, d, e, r = m["heads"], m["dim"], m["vdim"], rank or 5
            for name, n in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e)):
                lin(x + name, n, W)
            t[x + "q"] = (2 * t[x + "k"].float() + t[x + "q"].float()).to(torch.bfloat16)   # read-outs that do not cancel
            lin(x + "a1", r, W)
            lin(x + "a2", H * d, r, 2.0)
            uniform(x + "a2.b", H * d, -2, 6)
            put(x + "norm", e, scale=0.2, at=1.0)
            lin(x + "o", W, H * e)
        else:
            a = m["left"]
            H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for name, n in (("q", H * d), ("k", G * d), ("v", G * e), ("g", H)):
                lin(f"{x}left.{name}", n, W)
            put(x + "left.q.norm", d, scale=0.3, at=1.5)
            put(x + "left.k.norm", d, scale=0.3, at=1.5)
            lin(x + "left.o", W, H * e)
            a = m["right"]
            H, G, d, e, r, s = a["heads"], a["kv_heads"], a["dim"], a["vdim"], rank or 7, rank or 9
            for name, n in (("q", G * d), ("k", G * d), ("v", H * e)):
                lin(f"{x}right.{name}", n, W)
                put(f"{x}right.{name}.conv", n, a["conv"], scale=0.6)
            t[x + "right.q"] = (2 * t[x + "right.k"].float() + t[x + "right.q"].float()).to(torch.bfloat16)
            t[x + "right.q.conv"] = t[x + "right.k.conv"].clone()
            lin(x + "right.b", H, W)
            lin(x + "right.a1", r, W)
            lin(x + "right.a2", H * d, r)
            uniform(x + "right.dt_bias", H * d, -5, 1)
            uniform(x + "right.A_log", H, -2, 0.5)
            lin(x + "right.g1", s, W)
            lin(x + "right.g2", H * e, s)
            put(x + "right.norm", e, scale=0.2, at=1.0)
            lin(x + "right.o", W, H * e)
            put(x + "left.out", W, scale=0.2, at=1.0)
            put(x + "right.out", W, scale=0.2, at=1.0)
        if layer["mlp"]:
            f = layer["mlp"]["ff"]
            lin(p + "mlp.gate", f, W)
            lin(p + "mlp.up", f, W)
            lin(p + "mlp.down", W, f)
    return t


def tokens(c, n, seed):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


GLA = gla(heads=3, dim=40, vdim=24)
BOTH = parallel((6, 2, 32, 48, 0.2), (4, 2, 24, 40, 4))
MODELS = {
    "gla": config([GLA], 96, 128),
    "parallel": config([BOTH], 96, 128),
    "ff": config([(gla(1, 8, 8), 88)], 96, 128),
    "mixed": config([GLA, BOTH, gla(2, 64, 96, 8.0), (BOTH, None)], 112, 160, ff=96),
    # sizes that are no multiple of anything the kernels like, and no two alike
    "odd": config([(gla(3, 21, 35, 5.0), None), parallel((6, 3, 19, 22, 0.31), (6, 2, 13, 27, 3)), gla(2, 46, 9, 3.0),
                   (parallel((5, 5, 7, 50, 0.5), (3, 3, 67, 5, 7)), 53)], 90, 203, ff=41, eps=3e-4, embed=0.7, logits=1.3),
    # many heads: tiles of 64 columns; 128 key channels; one key head for all query heads
    "heads": config([gla(24, 128, 192), parallel((16, 1, 128, 128, 0.09), (20, 5, 128, 256, 4)), (gla(40, 24, 130), None),
                     (gla(48, 52, 128), None), (gla(10, 136, 258), None)], 256, 160, ff=128),
    # wider than the paged attention tiles and than one register block of the memories
    "big": config([gla(2, 200, 72), parallel((4, 2, 144, 160, 0.1), (2, 1, 300, 40, 5)), (gla(1, 512, 33), None)], 320, 333, ff=200),
    # rows of the residual beyond one and beyond both of its register blocks
    "wide_rows": config([gla(1, 16, 16), parallel((2, 1, 16, 16, 0.2), (1, 1, 16, 16, 2))], 2564, 64),
    "long_rows": config([gla(1, 16, 16), (parallel((2, 1, 16, 16, 0.2), (1, 1, 16, 16, 2)), 64)], 4100, 64),
    "ones": config([gla(1, 1, 1, 1.0), parallel((1, 1, 1, 1, 1.0), (1, 1, 1, 1, 1))], 16, 16, ff=1),
}
SERVED = config([GLA, BOTH, gla(2, 64, 96, 8.0)], 112, 160, ff=64)

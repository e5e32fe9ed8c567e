"""Plain implementation of the layer-list decoder (the Sinotar design): TEST INFRASTRUCTURE ONLY.

One function per mechanism, written token by token where the mechanism is a recurrence and as dense
matrices where it is not, in the precision of its inputs (the tests use float64 or float32).  It shares
no code with monoserve_b200: weights come in as a mapping from tensor name to tensor, the shape as the
parsed config.json.
"""
import math

import torch


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def over_rms(x, eps):
    """Each row divided by its root mean square, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, w, eps):
    return over_rms(x, eps) * (1 + w)


def log_sigmoid(z):
    return torch.minimum(z, torch.zeros_like(z)) - torch.log1p(torch.exp(-z.abs()))


def softplus(z):
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def silu(z):
    return z / (1 + torch.exp(-z))


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n] (last column: the current token), zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    return sum(padded[j:j + T] * taps[:, j] for j in range(n)) + bias


def rotate_pairs(x, pos, base):
    """x [..., T, dims] with (2i, 2i + 1) as pair i, angle pos * base^(-2 i / dims)."""
    dims = x.shape[-1]
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    a = pos.double()[:, None] * f[None]
    c, s = a.cos().to(x.dtype), a.sin().to(x.dtype)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def selective_scan(x, dt, A, B, C, D, state=None):
    """x, dt [T, c]; A [c, n]; B, C [T, n]; D [c].  Returns (y [T, c], final state [c, n])."""
    S = torch.zeros_like(A) if state is None else state.clone()
    y = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None]
        y.append(S @ C[t] + D * x[t])
    return torch.stack(y), S


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, e], log gates i, f [T, H].  Returns o [T, H, e]."""
    T, H, d = q.shape
    S, n, m = q.new_zeros(H, d, v.shape[-1]), q.new_zeros(H, d), q.new_zeros(H)
    out = []
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        dot = (n * q[t]).sum(-1)
        den = torch.maximum(dot.abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][:, :, None]).sum(1) / den[:, None])
    return torch.stack(out)


def mamba1(h, p, mixer, eps):
    inner, dt_rank, state = mixer["inner"], mixer["dt_rank"], mixer["state"]
    xz = h @ p["in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, p["conv"], p["conv.b"]))
    r = x @ p["x"].T
    dt, B, C = r[:, :dt_rank], r[:, dt_rank:dt_rank + state], r[:, dt_rank + state:]
    dt = softplus(dt @ p["dt"].T + p["dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(p["A_log"]), B, C, p["D"])
    return (y * silu(z)) @ p["o"].T


def latent_attention(h, p, mixer, eps):
    T, H, d, r, e, kvr = h.shape[0], mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    pos = torch.arange(T)
    base = mixer["rot"]["base"]
    q = (h @ p["q"].T).view(T, H, d + r).transpose(0, 1)
    c = h @ p["dkv"].T
    kr = rotate_pairs(c[:, kvr:], pos, base)
    c = over_rms(c[:, :kvr], eps) * p["dkv.norm"]
    k = (c @ p["uk"].T).view(T, H, d).transpose(0, 1)
    v = (c @ p["uv"].T).view(T, H, e).transpose(0, 1)
    qr = rotate_pairs(q[..., d:], pos, base)
    s = (q[..., :d] @ k.transpose(1, 2) + qr @ kr.T) * mixer["scale"]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    o = s.softmax(-1) @ v
    return o.transpose(0, 1).reshape(T, H * e) @ p["o"].T


def mlstm(h, p, mixer, eps):
    T, H, d, e, cap = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"], mixer["gate_cap"]
    q = (h @ p["q"].T).view(T, H, d) * d ** -0.5
    k, v = (h @ p["k"].T).view(T, H, d), (h @ p["v"].T).view(T, H, e)
    i = cap * torch.tanh((h @ p["i"].T + p["i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ p["f"].T + p["f.b"]) / cap))
    o = over_rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * e)
    g = h @ p["g"].T
    return (o * p["norm"] / (1 + torch.exp(-g))) @ p["o"].T


MIXERS = {"mamba1": mamba1, "latent_attention": latent_attention, "mlstm": mlstm}


def gated_ffn(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def layer_order(config):
    """Layer numbers in the order they run: the looped span repeated, the rest once."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


@torch.no_grad()
def model_logits(config, weights, tokens, dtype=torch.float64, runs=None, rows=None, jitter=0.0):
    """Logits [T, vocab] of one sequence.  runs (a list) receives the summed streams after every layer run;
    rows: only these positions' logits.  jitter: every sublayer's input and output is multiplied by 1 + up to this much at
    random, which shows how far rounding of that size carries."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    streams = [x] * config["streams"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}

    gen = torch.Generator().manual_seed(0)

    def shake(x):
        return x * (1 + jitter * (2 * torch.rand(x.shape, generator=gen, dtype=torch.float64) - 1)) if jitter else x

    def mixed(streams, hc, f):
        u = sum(a * x for a, x in zip(hc["in"], streams))
        y = shake(f(u))
        return [sum(hc["mix"][s, t] * streams[s] for s in range(len(streams))) + hc["out"][t] * y
                for t in range(len(streams))]

    for l in layer_order(config):
        spec, p = config["layers"][l], sub(f"l{l}.")
        mix = sub(f"l{l}.mix.")
        streams = mixed(streams, sub(f"l{l}.hc1."),
                        lambda u: MIXERS[spec["type"]](shake(norm_around_one(u, p["norm1"], eps)), mix, spec["mixer"], eps))
        if spec.get("mlp"):
            streams = mixed(streams, sub(f"l{l}.hc2."),
                            lambda u: gated_ffn(shake(norm_around_one(u, p["norm2"], eps)), sub(f"l{l}.mlp.")))
        if runs is not None:
            runs.append(sum(streams))
    x = sum(streams)
    if rows is not None:
        x = x[torch.as_tensor(rows)]
    return norm_around_one(x, w["final.norm"], eps) @ w["head"].T

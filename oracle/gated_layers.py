"""Plain implementation of the Teganex design (gated linear attention layers, and layers with attention and a gated delta
rule side by side): TEST INFRASTRUCTURE ONLY.

One function per mechanism, recurrences token by token, attention as a dense matrix, in the precision of the inputs (the
tests use float64 or float32).  It shares no code with monoserve_b200: weights come in as a mapping from tensor name to
tensor, the shape as the parsed config.json.
"""
import torch

from oracle.layer_list import causal_conv, over_rms, silu, softplus


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def unit(x, floor=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + floor)


def grouped_attention(q, k, v, scale):
    """Causal softmax attention; q [T, H, d], k [T, G, d], v [T, G, e] with H / G query heads on each key head."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T * scale).masked_fill(later, float("-inf"))
        out.append(s.softmax(-1) @ v[:, h // per])
    return torch.stack(out, 1)


def linear_memory(q, k, v, decay, state=None):
    """S <- diag(decay) S + k v^T, o = S^T q; q, k, decay [T, H, d], v [T, H, e].  Returns (o [T, H, e], S [H, d, e])."""
    T, H, d = q.shape
    S = q.new_zeros(H, d, v.shape[-1]) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def delta_memory(q, k, v, beta, decay, state=None):
    """S <- diag(decay) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q; beta [T, H], the rest as above."""
    T, H, d = q.shape
    S = q.new_zeros(H, d, v.shape[-1]) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def gla_decay(z, tau):
    return sigmoid(z) ** (1 / tau)


def delta_decay(z, A_log, heads):
    """z [T, heads * d] with its bias -> [T, heads, d]."""
    z = softplus(z).view(z.shape[0], heads, -1)
    return torch.exp(-torch.exp(A_log)[:, None] * z)


def attention_branch(h, p, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = over_rms((h @ p["q"].T).view(T, H, d), eps) * p["q.norm"]
    k = over_rms((h @ p["k"].T).view(T, G, d), eps) * p["k.norm"]
    o = grouped_attention(q, k, (h @ p["v"].T).view(T, G, e), m["scale"])
    o = o * sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(T, H * e) @ p["o"].T


def delta_branch(h, p, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ p[n].T, p[n + ".conv"], 0)) for n in "qkv")
    each = lambda x: unit(x.view(T, G, d)).repeat_interleave(H // G, 1)  # noqa: E731
    decay = delta_decay(h @ p["a1"].T @ p["a2"].T + p["dt_bias"], p["A_log"], H)
    o, _ = delta_memory(each(q) * d ** -0.5, each(k), v.view(T, H, e), sigmoid(h @ p["b"].T), decay)
    o = over_rms(o, eps) * p["norm"] * sigmoid(h @ p["g1"].T @ p["g2"].T).view(T, H, e)
    return o.reshape(T, H * e) @ p["o"].T


def gla(h, p, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ p["q"].T).view(T, H, d) * d ** -0.5, (h @ p["k"].T).view(T, H, d), (h @ p["v"].T).view(T, H, e)
    decay = gla_decay(h @ p["a1"].T @ p["a2"].T + p["a2.b"], m["tau"]).view(T, H, d)
    o, _ = linear_memory(q, k, v, decay)
    o = (over_rms(o, eps) * p["norm"]).reshape(T, H * e)
    return (o * silu(h @ p["g"].T)) @ p["o"].T


def below(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel(h, p, m, eps):
    left = attention_branch(h, below(p, "left."), m["left"], eps)
    right = delta_branch(h, below(p, "right."), m["right"], eps)
    return 0.5 * (over_rms(left, eps) * p["left.out"] + over_rms(right, eps) * p["right.out"])


MIXERS = {"gla": gla, "parallel": parallel}


def gated_ffn(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


@torch.no_grad()
def model_logits(config, weights, tokens, dtype=torch.float64, runs=None, rows=None, jitter=0.0):
    """Logits [T, vocab] of one sequence.  runs (a list) receives the residual after every layer; rows: only these positions'
    logits.  jitter: every sublayer's input and output is multiplied by 1 + up to this much at random, which shows how far
    rounding of that size carries."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    gen = torch.Generator().manual_seed(0)

    def shake(x):
        return x * (1 + jitter * (2 * torch.rand(x.shape, generator=gen, dtype=torch.float64) - 1)) if jitter else x

    x = w["embed"][torch.as_tensor(tokens)] * config["embedding"]["scale"] + w["pos"][:len(tokens)]
    for l, spec in enumerate(config["layers"]):
        p = below(w, f"l{l}.")
        norm = lambda x, name: over_rms(x, eps) * p[name]  # noqa: B023, E731
        x = x + norm(shake(MIXERS[spec["type"]](shake(norm(x, "norm1")), below(p, "mix."), spec["mixer"], eps)), "norm1b")
        if spec["mlp"]:
            x = x + norm(shake(gated_ffn(shake(norm(x, "norm2")), below(p, "mlp."))), "norm2b")
        if runs is not None:
            runs.append(x)
    if rows is not None:
        x = x[torch.as_tensor(rows)]
    return over_rms(x, eps) * w["final.norm"] @ w["head"].T * config["logit_scale"]

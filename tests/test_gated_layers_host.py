"""Host side of the Teganex design without a GPU: configuration, stacked projections, tile lists, the registry; and the plain
implementation the GPU tests compare with, against closed forms."""
import json
import types

import numpy as np
import pytest
import torch

from oracle import gated_layers as oracle
from tests import gated_models as gm
from tests import layer_list_models as lm
from tests.test_layer_list_host import POS0, REQUESTS, fields, lane


def test_config_is_read_with_every_branch():
    from monoserve_b200.layer_list import read_config
    c = gm.MODELS["odd"]
    cfg = read_config(c)
    assert [x.kind for x in cfg.layers] == ["gla", "parallel", "gla", "parallel"] and cfg.order == [0, 1, 2, 3]
    assert [x.ff for x in cfg.layers] == [0, 41, 41, 53]
    assert (cfg.model_type, cfg.hidden, cfg.vocab, cfg.eps, cfg.f32, cfg.streams) == ("teganex", 90, 203, 3e-4, False, 1)
    assert (cfg.embed_scale, cfg.logit_scale, cfg.max_positions) == (0.7, 1.3, 512)
    assert (cfg.layers[0].m.tau, cfg.layers[1].m.left.scale, cfg.layers[1].m.right.conv) == (5.0, 0.31, 3)
    assert read_config(c, "float32").f32


@pytest.mark.parametrize("layer,change,error", [
    (0, dict(type="mlstm"), NotImplementedError), (0, dict(type="mamba1"), NotImplementedError),
    (0, dict(mixer=dict(heads=1, dim=520, vdim=8, tau=1.0)), NotImplementedError),
    (1, dict(mixer=dict(lm.copy_of(gm.BOTH[1]), left=dict(gm.BOTH[1]["left"], dim=516))), NotImplementedError),
    (1, dict(mixer=dict(lm.copy_of(gm.BOTH[1]), left=dict(gm.BOTH[1]["left"], kv_heads=4))), ValueError),
    (1, dict(mixer=dict(lm.copy_of(gm.BOTH[1]), right=dict(gm.BOTH[1]["right"], conv=9))), NotImplementedError),
    (1, dict(mixer=dict(lm.copy_of(gm.BOTH[1]), right=dict(gm.BOTH[1]["right"], kv_heads=3))), ValueError),
    (0, dict(mlp=dict(kind="routed", ff=8)), NotImplementedError)])
def test_config_refuses_what_the_kernels_do_not_take(layer, change, error):
    from monoserve_b200.layer_list import read_config
    c = lm.copy_of(gm.MODELS["mixed"])
    c["layers"][layer].update(change)
    with pytest.raises(error):
        read_config(c)


def test_registry_finds_the_family(tmp_path):
    from monoserve_b200 import registry
    from monoserve_b200.layer_list import LayerListLane, read_config
    cfg = read_config(gm.SERVED)
    assert registry.lane_class(cfg) is LayerListLane
    c = gm.SERVED
    lm.write(str(tmp_path), c, gm.tensors(c, 2))
    with open(tmp_path / "config.json") as f:
        back = json.load(f)
    assert back == c and [x.matches(back) for x in registry.FAMILIES] == [False, True]


def test_stacked_projections_start_on_eight_columns():
    from monoserve_b200.gated_mixers import GatedDelta, GroupedAttention, Stack
    c = gm.MODELS["odd"]
    t = gm.tensors(c, 1)
    g = lambda n: t["l1.mix." + n]  # noqa: E731
    blocks = GatedDelta.blocks(g) + GroupedAttention.blocks(g)
    s = Stack(blocks)
    assert s.rows.shape == (s.n, 90) and len(s.at) == len(blocks) == 8
    used = torch.zeros(s.n, dtype=torch.bool)
    for name, w in blocks:
        at = s.at[name]
        assert at % 8 == 0 and torch.equal(s.rows[at:at + len(w)], w.float()) and not used[at:at + len(w)].any()
        used[at:at + len(w)] = True
    assert not s.rows[~used].any()
    m = types.SimpleNamespace(**c["layers"][1]["mixer"]["right"])
    assert dict(blocks)["right.qkv"].shape[0] == GatedDelta.channels(m) == 2 * 2 * 13 + 6 * 27


@pytest.mark.parametrize("heads,dim,e", [(3, 40, 24), (24, 128, 192), (40, 24, 130), (1, 512, 33), (2, 64, 64), (1, 1, 1), (48, 52, 128)])
def test_memory_tiles_cover_rows_heads_and_columns_once(heads, dim, e):
    from monoserve_b200.gated_mixers import K_GATED, K_GATED_STEP, gated_columns, gated_tiles, step_columns
    from monoserve_b200.layer_list import _Batch
    slot_of = {row: slot for row0, n, slot in REQUESTS for row in range(row0, row0 + n)}
    for f32, workers in ((False, 140), (True, 3)):
        b = _Batch(lane(), REQUESTS, POS0)
        width, step = gated_columns(REQUESTS, heads, dim, e, workers, f32), step_columns(dim)
        assert width in ((32, 64) if dim <= 128 else (16, 32, 64) if dim <= 256 else (16,)) and not (f32 and width == 64)
        seen = np.zeros((107, heads, e), int)
        t = fields(gated_tiles(b, heads, dim, e, workers, f32))
        of_row = {}
        for k, row, a, what, slot, cols in zip(t["kind"], t["i0"], t["i1"], t["i2"], t["i3"], t["a1"]):
            assert slot_of[row] == slot
            if k == K_GATED:
                head, block = what & 0xFFFF, what >> 16
                assert cols == width and slot_of[row + a - 1] == slot
                seen[row:row + a, head, block * width:(block + 1) * width] += 1
            else:
                assert k == K_GATED_STEP
                of_row[row] = of_row.get(row, 0) + 1
                blocks = -(-e // step)
                for v in range(what, what + a):
                    seen[row, v // blocks, v % blocks * step:(v % blocks + 1) * step] += 1
        assert (seen == 1).all()
        assert all(n <= max(1, workers // 2) for n in of_row.values()) and len(of_row) == 2


def test_wide_memory_tiles_are_used_where_they_save_a_round():
    from monoserve_b200.gated_mixers import gated_columns
    assert gated_columns([(0, 75, 0)], 24, 128, 192, 140) == 64     # 144 tiles of 32 columns are two rounds, 72 of 64 are one
    assert gated_columns([(0, 75, 0)], 24, 128, 128, 140) == 32     # 96 tiles are one round either way
    assert gated_columns([(0, 75, 0)], 24, 192, 192, 140) == 64     # more rows: three rounds of 16 columns, two of 32, one of 64
    assert gated_columns([(0, 75, 0)], 2, 192, 192, 140) == 16      # one round of any
    assert gated_columns([(0, 75, 0)], 24, 300, 192, 140) == 16
    assert gated_columns([(0, 75, 0)], 400, 128, 32, 140) == 32     # a head has no more


def test_conv_tiles_name_their_request_length():
    from monoserve_b200.layer_list import _Batch
    tiles = _Batch(lane(), REQUESTS, POS0).conv_tiles(1500)
    rows = {row0: n for row0, n, _ in REQUESTS}
    assert (tiles[:, 5].astype(int) == [rows[r] for r in fields(tiles)["i0"]]).all()


def test_attention_takes_the_tiles_it_fits():
    from monoserve_b200.gated_mixers import GroupedAttention as G
    m = lambda H, G_, d, e: types.SimpleNamespace(heads=H, kv_heads=G_, dim=d, vdim=e)  # noqa: E731
    bf, f32 = types.SimpleNamespace(f32=False), types.SimpleNamespace(f32=True)
    for args, page, want in (((6, 1, 64, 128), 16, True), ((6, 1, 64, 128), 24, False), ((6, 1, 129, 8), 16, False),
                             ((6, 1, 8, 130), 16, False), ((256, 1, 64, 64), 16, False), ((256, 2, 64, 64), 64, True)):
        assert G.tiled(bf, m(*args), page) == want and not G.tiled(f32, m(*args), page)
        d, e = G.widths(bf, m(*args), page)
        assert d % 8 == e % 8 == 0 and d >= args[2] and e >= args[3] and (not want or d == e == 128)


# ---------------------------------------------------------------------------------------------- the plain implementation
def rnd(g, *shape):
    return torch.randn(*shape, generator=g, dtype=torch.float64)


def test_oracle_memories_against_closed_forms():
    g = torch.Generator().manual_seed(0)
    T, H, d, e = 9, 2, 5, 3
    q, k, v, a = rnd(g, T, H, d), rnd(g, T, H, d), rnd(g, T, H, e), torch.rand(T, H, d, generator=g, dtype=torch.float64)
    o, S = oracle.linear_memory(q, k, v, a)
    for t in range(T):
        want = sum(torch.einsum("hd,hd,hd,he->he", q[t], a[s + 1:t + 1].prod(0), k[s], v[s]) for s in range(t + 1))
        assert torch.allclose(o[t], want)
    # the delta rule as one linear system per head: u = beta (v - A u), A_ts = k_t . prod(a) k_s for s < t
    k, beta = oracle.unit(k), torch.rand(T, H, generator=g, dtype=torch.float64)
    o, S = oracle.delta_memory(q, k, v, beta, a)
    for h in range(H):
        dots = torch.zeros(T, T, dtype=torch.float64)
        reads = torch.zeros(T, T, dtype=torch.float64)
        for t in range(T):
            for s in range(t + 1):
                w = a[s + 1:t + 1, h].prod(0) * k[s, h]
                dots[t, s] = 0 if s == t else (k[t, h] * w).sum()
                reads[t, s] = (q[t, h] * w).sum()
        u = torch.linalg.solve(torch.eye(T, dtype=torch.float64) + beta[:, h, None] * dots, beta[:, h, None] * v[:, h])
        assert torch.allclose(o[:, h], reads @ u)
    # split in two, carrying the state
    first, S1 = oracle.delta_memory(q[:4], k[:4], v[:4], beta[:4], a[:4])
    second, S2 = oracle.delta_memory(q[4:], k[4:], v[4:], beta[4:], a[4:], S1)
    assert torch.allclose(torch.cat([first, second]), o) and torch.allclose(S2, S)


def test_oracle_attention_and_decays():
    g = torch.Generator().manual_seed(1)
    q, k, v = rnd(g, 6, 4, 3), rnd(g, 6, 2, 3), rnd(g, 6, 2, 5)
    o = oracle.grouped_attention(q, k, v, 0.7)
    w = torch.exp(0.7 * (k[:4, 1] @ q[3, 2]))
    assert torch.allclose(o[3, 2], (w[:, None] * v[:4, 1]).sum(0) / w.sum()) and torch.allclose(o[0], v[0].repeat_interleave(2, 0))
    z = rnd(g, 4, 6)
    assert torch.allclose(oracle.gla_decay(z, 16.0), torch.exp(torch.nn.functional.logsigmoid(z) / 16))
    A = rnd(g, 2)
    want = torch.exp(-torch.exp(A)[None, :, None] * torch.nn.functional.softplus(z).view(4, 2, 3))
    assert torch.allclose(oracle.delta_decay(z, A, 2), want)


def test_four_tokens_at_a_time_is_the_delta_rule():
    """The identity the prefill tile computes by (four tokens per step, dot products between keys and queries as numbers)."""
    g = torch.Generator().manual_seed(2)
    d, e = 6, 3
    q, k, v, beta, a = rnd(g, 4, d), rnd(g, 4, d), rnd(g, 4, e), torch.rand(4, generator=g, dtype=torch.float64), \
        torch.rand(4, d, generator=g, dtype=torch.float64)
    S0 = rnd(g, d, e)
    want, S_want = oracle.delta_memory(q[:, None], k[:, None], v[:, None], beta[:, None], a[:, None], S0[None])
    c = torch.cumprod(a, 0)
    behind = lambda j, i: a[j + 1:i + 1].prod(0)  # noqa: E731
    u = []
    for i in range(4):
        p = S0.T @ (c[i] * k[i]) + sum(u[j] * (k[i] * behind(j, i) * k[j]).sum() for j in range(i))
        u.append(beta[i] * (v[i] - p))
        o = S0.T @ (c[i] * q[i]) + sum(u[j] * (q[i] * behind(j, i) * k[j]).sum() for j in range(i + 1))
        assert torch.allclose(o, want[i, 0])
    S = c[3][:, None] * S0 + sum((behind(j, 3) * k[j])[:, None] * u[j][None] for j in range(4))
    assert torch.allclose(S, S_want[0])


def test_oracle_shows_planted_mistakes():
    """The comparisons of the GPU tests notice each of these in the oracle itself."""
    from tests.test_gpu_layer_list import FLOOR, error
    c, toks = gm.MODELS["mixed"], gm.tokens(gm.MODELS["mixed"], 40, 3)
    t = gm.tensors(c, 4)
    ref = oracle.model_logits(c, t, toks)

    def with_changed(name, f):
        keep = getattr(oracle, name)
        setattr(oracle, name, f(keep))
        try:
            return oracle.model_logits(c, t, toks)
        finally:
            setattr(oracle, name, keep)

    late = lambda keep: lambda x, w, b: keep(torch.cat([x[:1], x[:-1]]), w, b)  # noqa: E731
    lost = lambda keep: lambda *x: (torch.cat([keep(*(v[:20] for v in x))[0], keep(*(v[20:] for v in x))[0]]), None)  # noqa: E731
    blind = lambda keep: lambda q, k, v, s: keep(q, torch.cat([k[:1], k[:-1]]), v, s)  # noqa: E731
    for name, f in (("causal_conv", late), ("linear_memory", lost), ("delta_memory", lost), ("grouped_attention", blind),
                    ("gla_decay", lambda keep: lambda z, tau: keep(z, 2 * tau)), ("unit", lambda keep: lambda x: keep(x, 30.0))):
        assert error(with_changed(name, f), ref) > 3 * FLOOR["bfloat16"], name
    moved = dict(t, pos=torch.roll(t["pos"], 1, 0))
    assert error(oracle.model_logits(c, moved, toks), ref) > 3 * FLOOR["bfloat16"]

"""Host side of the layer-list decoders (Sinotar) without a GPU: configuration, layer order, tile shapes, tile lists, the
model registry; and the plain implementation the GPU tests compare with, against closed forms."""
import json
import types

import numpy as np
import pytest
import torch

from oracle import layer_list as oracle
from tests import layer_list_models as lm


def lane(workers=140):
    return types.SimpleNamespace(fab=types.SimpleNamespace(num_workers=workers), items_per=lambda n: 4)


def fields(tiles):
    low, high = np.uint64(0xFFFFFFFF), np.uint64(32)
    return dict(kind=(tiles[:, 0] & np.uint64(0xFFFF)).astype(int), i0=(tiles[:, 1] & low).astype(int), i1=(tiles[:, 1] >> high).astype(int),
                i2=(tiles[:, 2] & low).astype(int), i3=(tiles[:, 2] >> high).astype(int), a1=tiles[:, 4].astype(int))


def test_config_is_read_with_every_branch():
    from monoserve_b200.layer_list import read_config
    cfg = read_config(lm.ODD)
    assert [x.kind for x in cfg.layers] == ["mamba1", "latent_attention", "mlstm", "mamba1"]
    assert cfg.order == [0, 1, 2, 1, 2, 1, 2, 3] == oracle.layer_order(lm.ODD)
    assert [x.ff for x in cfg.layers] == [41, 53, 0, 41]
    assert (cfg.hidden, cfg.vocab, cfg.streams, cfg.eps, cfg.f32) == (90, 203, 5, 3e-4, False)
    plain = read_config(lm.WIDE, "float32")
    assert plain.order == [0, 1, 2, 3] and plain.f32 and [x.ff for x in plain.layers] == [0, 700, 700, 0]
    assert [x.ff for x in read_config(lm.ALONE["memory"]).layers] == [0]


@pytest.mark.parametrize("change", [
    dict(type="other"), dict(mlp=dict(kind="routed", ff=8)), dict(mixer=dict(lm.SCAN[1], conv=9)), dict(mixer=dict(lm.SCAN[1], state=200))])
def test_config_refuses_what_the_kernels_do_not_take(change):
    from monoserve_b200.layer_list import read_config
    c = json.loads(json.dumps(lm.ALONE["scan"]))
    c["layers"][0].update(change)
    with pytest.raises(NotImplementedError):
        read_config(c)


def test_registry_finds_the_family(tmp_path):
    from monoserve_b200 import registry
    from monoserve_b200.layer_list import LayerListLane, read_config
    from monoserve_b200.model import ModelLane
    assert registry.lane_class(read_config(lm.MIXED)) is LayerListLane
    assert registry.lane_class(types.SimpleNamespace(model_type="qwen3_moe")) is ModelLane
    assert registry.lane_class(types.SimpleNamespace(), default="stand-in") == "stand-in"
    with open(tmp_path / "config.json", "w") as f:
        json.dump(dict(architecture="unheard of"), f)
    with pytest.raises(NotImplementedError, match="unheard of"):
        registry.load(str(tmp_path))


def test_checkpoint_folder_round_trip(tmp_path):
    from monoserve_b200.layer_list import read_tensors
    t = lm.tensors(lm.ODD, 1)
    lm.write(str(tmp_path), lm.ODD, t)
    back = read_tensors(str(tmp_path))
    assert back.keys() == t.keys() and all(torch.equal(back[k], v) for k, v in t.items())


def test_attention_tile_shapes_fit_the_worker():
    from monoserve_b200.layer_list import RING_BYTES, direct_buffers, latent_tile
    for heads in (1, 3, 5, 16, 17, 40, 128):
        for dim, rot, vdim, rank in ((128, 64, 128, 512), (24, 8, 40, 72), (64, 32, 96, 320), (19, 6, 21, 45), (64, 32, 64, 768)):
            m = types.SimpleNamespace(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank)
            for tokens in (1, 2, 7, 500):
                shape = latent_tile(m, 16, tokens)
                if shape is None:
                    assert rank >= 768
                    continue
                tok, hg, buffers = shape
                cols = next(n for n in (16, 32, 64) if n >= tok * hg)
                chunks = -(-(rank + rot) // 64)
                assert 1 <= tok <= tokens and tok * hg <= 64 and 1 <= hg <= heads
                assert cols * (chunks * 128 + 256) + buffers * chunks * 128 * 128 <= RING_BYTES
                assert 64 + -(-rank // 128) * cols <= 512     # TMEM columns
            assert latent_tile(m, 24, 1) is None and latent_tile(m, 4, 1) is None   # page sizes a key tile cannot be made of
            b = direct_buffers(m)
            nq = -(-dim // 64) + -(-rot // 64)
            assert (b == 0) == any(v % 8 for v in (dim, rot, vdim, rank)) and (nq * (1 + b) + -(-vdim // 64) + 2) * 16384 <= RING_BYTES


REQUESTS, POS0 = [(0, 70, 4), (70, 1, 1), (71, 33, 2), (104, 2, 7), (106, 1, 0)], [0, 9, 0, 64, 0]


def test_tile_lists_cover_rows_channels_columns_and_heads_once():
    from monoserve_b200.layer_list import K_CONV, K_MEMORY, K_MEMORY_STEP, K_SCAN, K_SCAN_STEP, _Batch
    b = _Batch(lane(), REQUESTS, POS0)
    slot_of = {row: slot for row0, n, slot in REQUESTS for row in range(row0, row0 + n)}
    for channels in (33, 1024, 1500):
        seen = np.zeros((107, channels), int)
        t = fields(b.conv_tiles(channels))
        for k, first, row, what, slot, c0 in zip(t["kind"], t["i0"], t["i1"], t["i2"], t["i3"], t["a1"]):
            rows, count = what & 0xFFFF, what >> 16
            assert k == K_CONV and slot_of[row] == slot == slot_of[row + rows - 1] and slot_of[first] == slot
            seen[row:row + rows, c0:c0 + count] += 1
        assert (seen == 1).all()
        seen[:] = 0
        t = fields(b.scan_tiles(channels))
        for k, row, a, c0, slot in zip(t["kind"], t["i0"], t["i1"], t["i2"], t["i3"]):
            rows, count = (a, 32) if k == K_SCAN else (1, a)
            assert k in (K_SCAN, K_SCAN_STEP) and (rows == 1) == (k == K_SCAN_STEP) and slot_of[row] == slot
            seen[row:row + rows, c0:min(channels, c0 + count)] += 1
        assert (seen == 1).all()
    for heads, e in ((3, 40), (2, 31), (8, 512), (1, 32)):
        blocks = e // 32 + 1
        seen = np.zeros((107, heads, blocks), int)
        t = fields(b.memory_tiles(heads, e))
        for k, row, a, what, slot in zip(t["kind"], t["i0"], t["i1"], t["i2"], t["i3"]):
            head, block = what & 0xFFFF, what >> 16
            rows, count = (a, 1) if k == K_MEMORY else (1, a)
            assert k in (K_MEMORY, K_MEMORY_STEP) and slot_of[row] == slot
            seen[row:row + rows, head, block:block + count] += 1
        assert (seen == 1).all()
    for heads, parts in ((5, 1), (5, 3), (16, 2)):
        seen = np.zeros((107, heads, parts), int)
        t = fields(b.attn_tiles(heads, parts))
        for row, what, part, total, slot in zip(t["i0"], t["i1"], t["i2"], t["i3"], t["a1"]):
            assert total == parts and slot_of[row] == slot
            seen[row, what & 0xFFFF:(what & 0xFFFF) + (what >> 16), part] += 1
        assert (seen == 1).all()
        seen[:] = 0
        t = fields(b.latent_tiles(heads, 3, 4, parts))
        for row, what, part, slot in zip(t["i0"], t["i1"], t["i2"], t["a1"]):
            rows, h0 = what & 0xFFFF, what >> 16
            assert {slot_of[r] for r in range(row, row + rows)} == {slot}
            seen[row:row + rows, h0:h0 + 4, part] += 1
        assert (seen == 1).all()


def test_whole_prompts_are_told_from_portions():
    from monoserve_b200.layer_list import _Batch
    whole, rest = _Batch(lane(), REQUESTS, POS0).split()
    assert whole == [REQUESTS[0], REQUESTS[2]] and rest.requests == [REQUESTS[1], REQUESTS[3], REQUESTS[4]]
    assert rest.spans() == [(70, 1), (104, 3)]
    items = fields(rest.item_tiles(61, 5))
    covered = np.concatenate([np.arange(a, a + n) for a, n in zip(items["i0"], items["i1"])])
    assert sorted(covered) == sorted(r * 5 + j for r in (70, 104, 105, 106) for j in range(5))
    assert _Batch(lane(), REQUESTS).split()[0] == []      # a decode step


def test_oracle_recurrences_against_closed_forms():
    g = torch.Generator().manual_seed(0)
    T, c, n = 9, 3, 4
    x, dt, B, C = (torch.randn(*s, generator=g, dtype=torch.float64) for s in ((T, c), (T, c), (T, n), (T, n)))
    dt, A, D = dt.abs(), -torch.rand(c, n, generator=g, dtype=torch.float64), torch.randn(c, generator=g, dtype=torch.float64)
    y, _ = oracle.selective_scan(x, dt, A, B, C, D)
    for t in range(T):
        want = D * x[t]
        for s in range(t + 1):
            decay = torch.exp(dt[s + 1:t + 1].sum(0)[:, None] * A)
            want = want + ((decay * B[s] * C[t]).sum(-1)) * dt[s] * x[s]
        assert torch.allclose(y[t], want)
    H, d, e = 2, 5, 3
    q, k, v = (torch.randn(T, H, w, generator=g, dtype=torch.float64) for w in (d, d, e))
    i, f = torch.randn(T, H, generator=g, dtype=torch.float64), -torch.rand(T, H, generator=g, dtype=torch.float64)
    o = oracle.matrix_memory(q, k, v, i, f)
    for t in range(T):
        # without the running maximum: weights e^(i_s + sum of f after s), floor e^0 = 1 (m starts at 0)
        w = torch.stack([torch.exp(i[s] + f[s + 1:t + 1].sum(0)) for s in range(t + 1)])
        dots = torch.einsum("shd,hd->sh", k[:t + 1], q[t])
        m = torch.maximum(f[:t + 1].sum(0), torch.stack([i[s] + f[s + 1:t + 1].sum(0) for s in range(t + 1)]).max(0).values)
        den = torch.maximum((w * dots).sum(0).abs(), torch.ones(H, dtype=torch.float64)) + 1e-6 * torch.exp(m)
        assert torch.allclose(o[t], torch.einsum("sh,sh,she->he", w, dots, v[:t + 1]) / den[:, None])


def test_oracle_shows_planted_mistakes():
    """The comparisons of the GPU tests notice each of these in the oracle itself: a convolution off by one, a state that
    is lost between portions, interleaved pairs taken as halves, the last layer pass left out."""
    from tests.test_gpu_layer_list import FLOOR, error
    c, toks = lm.MIXED, lm.tokens(lm.MIXED, 40, 3)
    t = lm.tensors(c, 4)
    ref = oracle.model_logits(c, t, toks)

    def with_changed(name, f):
        keep = getattr(oracle, name)
        setattr(oracle, name, f(keep))
        try:
            return oracle.model_logits(c, t, toks)
        finally:
            setattr(oracle, name, keep)

    halves = lambda keep: lambda x, pos, base: keep(torch.cat([x[..., 0::2], x[..., 1::2]], -1), pos, base)  # noqa: E731
    late = lambda keep: lambda x, w, b: keep(torch.cat([x[:1], x[:-1]]), w, b)  # noqa: E731
    lost = lambda keep: lambda q, k, v, i, f: torch.cat([keep(q[:20], k[:20], v[:20], i[:20], f[:20]),  # noqa: E731
                                                        keep(q[20:], k[20:], v[20:], i[20:], f[20:])])
    for name, f in (("rotate_pairs", halves), ("causal_conv", late), ("matrix_memory", lost)):
        assert error(with_changed(name, f), ref) > 3 * FLOOR["bfloat16"], name
    short = dict(c, loop=dict(c["loop"], times=1))
    assert error(oracle.model_logits(short, t, toks), ref) > 3 * FLOOR["bfloat16"]

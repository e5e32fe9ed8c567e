"""Mixers with gated memories and grouped-query attention for the layer-list decoders (monoserve_b200/layer_list.py): gated
linear attention, and grouped-query attention beside a gated delta rule.

Every projection that reads a mixer's input is a row block of one stacked matrix, so a mixer starts with one GEMM whose
output columns are then read in place: `Stack` keeps where each block starts (multiples of eight columns, so that a block
can be a GEMM operand or a 16-byte vector load).
"""
import types

import numpy as np
import torch

from monoserve_b200 import _C
from monoserve_b200.attention import fabric_maps, fabric_tiles, plan_items
from monoserve_b200.fabric import tile_array
from monoserve_b200.lane_base import EPI_DECAY, _block, _retarget, up

K_HEAD_NORM = 58
K_DECAY, K_GATED, K_GATED_STEP, K_QKV, K_GROUPED_ATTN, K_HEAD_GATE = 67, 68, 69, 70, 71, 72
K_ATTN_PREFILL, K_ATTN_PLAN = 33, 44
MAX_GATED_DIM, MAX_CONV_TAPS, MAX_HEAD_COLUMNS = 512, 8, 512
PAD_HEAD, MAX_PLAN_ROWS, MAX_CHUNKS = 128, 256, 8   # of the paged attention tiles: head width, decode rows, key ranges of a row
QKV_ITEMS = 64


class Stack:
    """Row blocks of one stacked matrix: `at[name]` is the first column of a block in the product, `n` the columns."""

    def __init__(self, blocks):
        self.at, rows, n = {}, [], 0
        for name, t in blocks:
            self.at[name] = n
            pad = up(t.shape[0], 8) - t.shape[0]
            rows.append(torch.nn.functional.pad(t.float(), (0, 0, 0, pad)))
            n += t.shape[0] + pad
        self.n, self.rows = n, torch.cat(rows)


# ---------------------------------------------------------------------------------------------- shared pieces
def check_gated(i, m):
    if m["dim"] > MAX_GATED_DIM:
        raise NotImplementedError(f"layer {i}: gated memory of {m['dim']} key dimensions (to {MAX_GATED_DIM})")


def gated_state(m, slots):
    return torch.zeros(slots, m.heads, m.vdim, up(m.dim, 4), device="cuda")


def decay_stage(lane, p, prev, b, x, w, m, label):
    """expm1 of the log decays of every head and key channel, -coef softplus(x a2^T + bias), from their low-rank activations
    x [rows][w.rank]: the epilogue of the product, or in 32-bit a tile behind it."""
    n = m.heads * m.dim
    if not lane.cfg.f32:
        return lane.product(p, prev, x, w.a2, lane.decay, b.T, n, w.rank, label, epi=EPI_DECAY, bias=w.a_bias, coef=w.coef)
    s = lane.product(p, prev, x, w.a2, lane.decay, b.T, n, w.rank, label)
    args = lane._dev("DecayArgs", z=lane.decay.addr, bias=w.a_bias, coef=w.coef, ld=lane.decay.ld, n=n)
    s_d = p.stage(lane._rows(K_DECAY, args, b.T, lane._per(b.T)), label=label)
    p.after(s, s_d)
    return s_d


def place_decay(W, a2, bias, coef, dim):
    """a2 [heads * dim, rank] and bias as the decay stage takes them (the bias in fp32 for its tile, else the checkpoint's
    bf16 as a GEMM's), the heads' coefficients once per channel."""
    return types.SimpleNamespace(a2=W.mat(a2), a_bias=W.f32(bias) if W.cfg.f32 else bias.to(torch.bfloat16).contiguous().cuda(),
                                 coef=coef.float().repeat_interleave(dim).contiguous().cuda(), rank=a2.shape[1])


def gated_columns(requests, heads, dim, columns, workers, f32=False):
    """Columns of a portion's tile: the width whose rounds of tiles over the workers cost least, a tile of twice the columns
    costing about a third more."""
    widths = (32, 64) if dim <= 128 else (16, 32, 64) if dim <= 256 else (16,)
    portions = sum(1 for _, n, _ in requests if n > 1) * heads
    fit = [w for w in widths[:1 if f32 else None] if w == widths[0] or w <= up(columns, widths[0])]
    return min(fit, key=lambda w: -(-portions * -(-columns // w) // workers) * (4 / 3) ** widths.index(w))


def step_columns(dim):
    """Columns of one block of the one-token tile: its four warps hold 128 columns of up to 64 rows, 64 of up to 128, ..."""
    return next(c for rows, c in ((64, 128), (128, 64), (256, 32), (512, 16)) if dim <= rows)


def gated_tiles(b, heads, dim, e, workers, f32):
    """Portions: a tile per head and block of columns, the longest first; single tokens: each row's column blocks, counted
    through its heads, in as many tiles as leave no worker two."""
    def make():
        width = gated_columns(b.requests, heads, dim, e, workers, f32)
        h, c = np.meshgrid(np.arange(heads), np.arange(-(-e // width)), indexing="ij")
        out = [tile_array(K_GATED, i0=row0, i1=n, i2=h | (c << 16), i3=slot, a1=width)
               for row0, n, slot in sorted(b.requests, key=lambda q: -q[1]) if n > 1]
        ones = [(row0, slot) for row0, n, slot in b.requests if n == 1]
        if ones:
            row, slot = (np.array(v)[:, None] for v in zip(*ones))
            blocks = heads * -(-e // step_columns(dim))
            per = -(-blocks // min(blocks, max(1, workers // len(ones))))
            first = np.arange(0, blocks, per)[None]
            out.append(tile_array(K_GATED_STEP, i0=row, i1=np.minimum(per, blocks - first), i2=first, i3=slot))
        return np.concatenate(out)
    return b._once(("gated", heads, dim, e), make)


def memory_stage(lane, p, prev, b, m, group, q, k, v, ld, beta, ld_beta, state, unit, q_scale, label):
    mem = lane._dev("GatedMemoryArgs", q=q, k=k, v=v, beta=beta, decay=lane.decay.addr, state=state, out=lane.raw.addr,
                    tok_pos=lane.tok_pos, ld_qkv=ld, ld_beta=ld_beta, ld_decay=lane.decay.ld, heads=m.heads, group=group, d=m.dim,
                    e=m.vdim, f32=int(lane.cfg.f32), unit=unit, q_scale=q_scale)
    tiles = gated_tiles(b, m.heads, m.dim, m.vdim, lane.fab.num_workers, lane.cfg.f32)
    s = p.stage(_retarget(tiles, a0=mem.data_ptr()), label=label)
    for stage in prev:
        p.after(stage, s)
    return s


def head_norm_stage(lane, p, prev, T, m, g, norm, silu, label):
    nrm = lane._dev("HeadNormArgs", o=lane.raw.addr, g=g.addr, w=norm, out=lane.mix.addr, heads=m.heads, e=m.vdim, ld_g=g.ld,
                    ld_out=lane.mix.ld, f32=int(lane.cfg.f32), eps=lane.cfg.eps, w_head=0, silu=silu)
    s = p.stage(lane._rows(K_HEAD_NORM, nrm, T * m.heads, lane.items_per(T * m.heads)), label=label)
    for stage in prev:
        p.after(stage, s)
    return s


# ---------------------------------------------------------------------------------------------- gated linear attention
class GatedLinear:
    """S <- diag(sigmoid(z)^(1 / tau)) S + k v^T, o = S^T q with z = W_a2 W_a1 h + b; head norm, silu gate, W_o."""

    @staticmethod
    def check(i, m):
        check_gated(i, m)

    @staticmethod
    def place(W, w, m, g):
        w.stack = Stack([(n, g(n)) for n in ("q", "k", "v", "g", "a1")])
        w.in_, w.o, w.norm = W.mat(w.stack.rows), W.mat(g("o")), W.f32(g("norm"))
        # log of sigmoid(z)^(1 / tau) = -softplus(-z) / tau
        w.decay = place_decay(W, -g("a2"), -g("a2.b"), torch.full((m.heads,), 1.0 / m.tau), m.dim)

    @staticmethod
    def state(cfg, m, rows, slots, page):
        return dict(S=gated_state(m, slots))

    @staticmethod
    def sizes(m, w):
        return dict(proj=w.stack.n, mix=m.heads * m.vdim, decay=m.heads * m.dim, raw=m.heads * up(m.vdim, 4))

    @staticmethod
    def prepare(lane, layer, w, run_state):
        lane.weight_map(w.in_), lane.weight_map(w.o), lane.weight_map(w.decay.a2)
        lane.mix.maps(layer.m.heads * layer.m.vdim), lane.proj.view(w.stack.at["a1"]).maps(w.decay.rank)

    @staticmethod
    def build(lane, p, l, run, b, prev):
        m, w, T = lane.cfg.layers[l].m, lane.w.layers[l], b.T
        s = lane.product(p, prev, lane.h, w.in_, lane.proj, T, w.stack.n, lane.cfg.hidden, ("gla_in", run), out16=True)
        at = {name: lane.proj.view(col) for name, col in w.stack.at.items()}
        s_a = decay_stage(lane, p, s, b, at["a1"], w.decay, m, ("gla_decay", run))
        s_m = memory_stage(lane, p, [s_a], b, m, 1, at["q"].addr, at["k"].addr, at["v"].addr, lane.proj.ld, 0, 0,
                           lane.kv.runs[run]["S"], 0, m.dim ** -0.5, ("gla", run))
        s_n = head_norm_stage(lane, p, [s_m], T, m, at["g"], w.norm, 1, ("gla_norm", run))
        return lane.closing(p, s_n, lane.mix, w.o, T, m.heads * m.vdim, ("gla_o", run))


# ---------------------------------------------------------------------------------------------- the two sides of Parallel
class GroupedAttention:
    """Causal softmax attention, kv_heads key / value heads shared by groups of query heads, normed queries and keys, no
    rotation, one output gate per head.  Heads of up to 128 columns run on the paged attention tiles, padded to 128."""

    @staticmethod
    def check(i, m):
        if max(m["dim"], m["vdim"]) > MAX_HEAD_COLUMNS:
            raise NotImplementedError(f"layer {i}: heads of {m['dim']} and {m['vdim']} columns (to {MAX_HEAD_COLUMNS})")
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key heads")

    @staticmethod
    def tiled(cfg, m, page):
        """The tensor-core tiles take this layer."""
        return not cfg.f32 and max(m.dim, m.vdim) <= PAD_HEAD and m.heads // m.kv_heads <= 128 and page % 8 == 0 and 128 % page == 0

    @staticmethod
    def widths(cfg, m, page):
        """Columns of a head in the query and key rows, and in the value and output rows."""
        return (PAD_HEAD, PAD_HEAD) if GroupedAttention.tiled(cfg, m, page) else (up(m.dim, 8), up(m.vdim, 8))

    @staticmethod
    def blocks(g):
        return [("left." + n, g("left." + n)) for n in ("q", "k", "v", "g")]

    @staticmethod
    def place(W, m, g):
        return types.SimpleNamespace(o=W.mat(g("left.o")), q_norm=W.f32(g("left.q.norm")), k_norm=W.f32(g("left.k.norm")),
                                     out=W.f32(g("left.out")))

    @staticmethod
    def state(cfg, m, rows, page):
        d, e = GroupedAttention.widths(cfg, m, page)
        z = lambda n: torch.zeros(rows // page, page, m.kv_heads, n, device="cuda",  # noqa: E731
                                  dtype=torch.float32 if cfg.f32 else torch.bfloat16)
        return dict(k=z(d), v=z(e))

    @staticmethod
    def sizes(m):
        wide = max(PAD_HEAD, up(m.dim, 8)), max(PAD_HEAD, up(m.vdim, 8))
        return dict(gq=m.heads * wide[0], go=m.heads * wide[1], mix2=m.heads * m.vdim)

    @staticmethod
    def prepare(lane, m, st):
        """The operand block of the paged attention over this run's cache; its split workspace covers every plan: a part has
        at least its share of the total, so the rows of split items are at most the batch's own plus two rounds of tiles."""
        lane.mix2.maps(m.heads * m.vdim)
        if not GroupedAttention.tiled(lane.cfg, m, lane.kv.page):
            return
        H, T = m.heads, lane.T
        need = max(MAX_CHUNKS * min(T, MAX_PLAN_ROWS) * H, T * H + 256 * lane.fab.num_workers)
        if getattr(lane, "attn_ws_rows", 0) < need:
            lane.attn_ws, lane.attn_ws_rows = torch.zeros(need * 130, device="cuda"), need
            lane._keep.append(lane.attn_ws)
        q = lane.gq.t[:T * H * PAD_HEAD].view(T, H, PAD_HEAD)
        q_map, q_small, k_map, v_map = fabric_maps(lane.fab, q, st["k"], st["v"])
        lane.attn_blocks[st["k"].data_ptr()] = _block(
            "AttnArgs", q_map=q_map, q_map_small=q_small, k_map=k_map, v_map=v_map, out=lane.go.addr, ws_o=lane.attn_ws,
            ws_m=lane.attn_ws.data_ptr() + lane.attn_ws_rows * 512, block_table=lane.bt, req_info=lane.req_info,
            scale_log2=m.scale * 1.4426950408889634, bt_stride=lane.bt_stride, hq=H, hkv=m.kv_heads, group=H // m.kv_heads,
            max_chunks=MAX_CHUNKS, page_size=lane.kv.page)

    @staticmethod
    def build(lane, p, m, w, st, at, run, b, prev):
        H, G, T, f32, page = m.heads, m.kv_heads, b.T, int(lane.cfg.f32), lane.kv.page
        d, e = GroupedAttention.widths(lane.cfg, m, page)
        qkv = lane._dev("QkvArgs", q=at["left.q"].addr, k=at["left.k"].addr, v=at["left.v"].addr, q_norm=w.q_norm, k_norm=w.k_norm,
                        q_out=lane.gq.addr, k_cache=st["k"], v_cache=st["v"], tok_slot=lane.tok_slot, ld_x=lane.proj.ld, heads=H,
                        kv_heads=G, d=m.dim, e=m.vdim, ld_q=d, ld_k=d, ld_v=e, f32=f32, eps=lane.cfg.eps)
        items = T * (H + 2 * G)
        s = p.stage(lane._rows(K_QKV, qkv, items, min(QKV_ITEMS, max(8, up(-(-items // lane.fab.num_workers), 8)))), label=("qkv", run))
        p.after(prev, s)
        tiled = GroupedAttention.tiled(lane.cfg, m, page)
        if tiled and b.pos0 is not None:
            s = GroupedAttention.planned(lane, p, st, H, G, run, b, s)
        elif tiled and T <= MAX_PLAN_ROWS:
            s = GroupedAttention.stepped(lane, p, st, G, run, b, s)
        else:
            args = lane._dev("GroupedAttnArgs", q=lane.gq.addr, k_cache=st["k"], v_cache=st["v"], block_table=lane.bt,
                             out=lane.go.addr, tok_pos=lane.tok_pos, heads=H, kv_heads=G, d=m.dim, e=m.vdim, ld_q=d, ld_k=d, ld_v=e,
                             ld_out=e, page=page, bt_stride=lane.bt_stride, f32=f32, scale=m.scale)
            s_at = p.stage(_retarget(b.attn_tiles(H, 1, kind=K_GROUPED_ATTN), a0=args.data_ptr()), label=("attn", run))
            p.after(s, s_at)
            s = s_at
        gate = lane._dev("HeadGateArgs", g=at["left.g"].addr, out=lane.mix2.addr, heads=H, e=m.vdim, ld_in=e, ld_g=lane.proj.ld,
                         ld_out=lane.mix2.ld, f32=f32, **{"in": lane.go.addr})
        s_g = p.stage(lane._rows(K_HEAD_GATE, gate, T, lane._per(T)), label=("head_gate", run))
        p.after(s, s_g)
        return lane.closing(p, s_g, lane.mix2, w.o, T, H * m.vdim, ("attn_o", run), out=lane.y2)

    @staticmethod
    def planned(lane, p, st, H, G, run, b, prev):
        """Prompts and portions: the work list is made here."""
        def make():
            info = [(row0, pos0, n, pos0 + n) for (row0, n, _), pos0 in zip(b.requests, b.pos0)]
            items, merge, ws_rows = plan_items(info, H, G, sms=lane.fab.num_workers)
            assert ws_rows <= lane.attn_ws_rows, "attention split workspace too small"
            items[:, 0] = torch.tensor([slot for _, _, slot in b.requests], dtype=torch.int32)[items[:, 0].long()]
            return fabric_tiles(items, merge, 0, K_ATTN_PREFILL)
        item_tiles, merge_tiles = b._once(("plan", H, G), make)
        at = lane.attn_blocks[st["k"].data_ptr()].data_ptr()
        s = p.stage(_retarget(item_tiles, a0=at), label=("attn", run))
        p.after(prev, s)
        if len(merge_tiles):
            s_m = p.stage(_retarget(merge_tiles, a0=at), label=("attn_merge", run))
            p.after(s, s_m)
            s = s_m
        return s

    @staticmethod
    def stepped(lane, p, st, G, run, b, prev):
        """A decode step: a plan tile behind the embedding stage writes the step's items."""
        blob = lane.arena.put(bytes(_C.struct_layouts()["AttnPlanArgs"][0]))   # filled with the dynamic region
        s_plan = p.stage(lane._one(K_ATTN_PLAN, blob), label=("attn_plan", run))
        s_a, s_m = p.stage(label=("attn", run)), p.stage(label=("attn_merge", run))
        p.after(b.first, s_plan)
        p.after(s_plan, s_a)
        p.after(prev, s_a)
        p.after(s_a, s_m)
        b.plans.append((blob, dict(attn=lane.attn_blocks[st["k"].data_ptr()].data_ptr(), req_info=lane.req_info.data_ptr(), rows=b.T,
                                   hkv=G, stage_attn=s_a, stage_comb=s_m, workers=lane.fab.num_workers,
                                   row_req=lane.row_req.data_ptr()), b.T * G * (MAX_CHUNKS + 1)))
        return s_m


class GatedDelta:
    """q, k, v through a short convolution and silu, q and k as unit vectors per head; S <- diag(a) S,
    u = sigmoid(b) (v - S^T k), S <- S + k u^T, o = S^T q with log a = -exp(A_log) softplus(W_a2 W_a1 h + dt); head norm,
    sigmoid gate, W_o.  Groups of value heads share a query / key head."""

    @staticmethod
    def check(i, m):
        check_gated(i, m)
        if not 1 <= m["conv"] <= MAX_CONV_TAPS:
            raise NotImplementedError(f"layer {i}: {m['conv']} taps (to {MAX_CONV_TAPS})")
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {i}: {m['heads']} value heads over {m['kv_heads']} key heads")

    @staticmethod
    def channels(m):
        return 2 * m.kv_heads * m.dim + m.heads * m.vdim

    @staticmethod
    def blocks(g):
        qkv = torch.cat([g("right." + n) for n in "qkv"])   # one block: the convolution runs over all of its channels
        return [("right.qkv", qkv)] + [("right." + n, g("right." + n)) for n in ("b", "a1", "g1")]

    @staticmethod
    def place(W, m, g):
        g_ = lambda n: g("right." + n)  # noqa: E731
        return types.SimpleNamespace(
            o=W.mat(g_("o")), norm=W.f32(g_("norm")), out=W.f32(g_("out")), conv=W.f32(torch.cat([g_(f"{n}.conv") for n in "qkv"])),
            decay=place_decay(W, g_("a2"), g_("dt_bias"), torch.exp(g_("A_log").float()), m.dim), g2=W.mat(g_("g2")),
            gate_rank=g_("g1").shape[0])

    @staticmethod
    def state(m, slots):
        return dict(S=gated_state(m, slots), tail=torch.zeros(slots, max(1, m.conv - 1), GatedDelta.channels(m), device="cuda"))

    @staticmethod
    def sizes(m):
        return dict(act=GatedDelta.channels(m), mix=m.heads * m.vdim, gate=m.heads * m.vdim, decay=m.heads * m.dim,
                    raw=m.heads * up(m.vdim, 4))

    @staticmethod
    def prepare(lane, m, w, at):
        for t in (w.g2, w.o, w.decay.a2):
            lane.weight_map(t)
        lane.mix.maps(m.heads * m.vdim), lane.proj.view(at["right.g1"]).maps(w.gate_rank)
        lane.proj.view(at["right.a1"]).maps(w.decay.rank)

    @staticmethod
    def build(lane, p, m, w, st, at, run, b, prev):
        T, f32, kd = b.T, int(lane.cfg.f32), m.kv_heads * m.dim
        conv = lane._dev("ConvArgs", x=at["right.qkv"].addr, tail=st["tail"], w=w.conv, out=lane.act.addr, tok_pos=lane.tok_pos,
                         ld_x=lane.proj.ld, ld_out=lane.act.ld, channels=GatedDelta.channels(m), taps=m.conv, f32=f32, advance=1)
        s_c = p.stage(_retarget(b.conv_tiles(GatedDelta.channels(m)), a0=conv.data_ptr()), label=("delta_conv", run))
        p.after(prev, s_c)
        s_a = decay_stage(lane, p, prev, b, at["right.a1"], w.decay, m, ("delta_decay", run))
        s_g = lane.product(p, prev, at["right.g1"], w.g2, lane.gate, T, m.heads * m.vdim, w.gate_rank, ("delta_gate", run), out16=True)
        s_m = memory_stage(lane, p, [s_c, s_a], b, m, m.heads // m.kv_heads, lane.act.addr, lane.act.view(kd).addr,
                           lane.act.view(2 * kd).addr, lane.act.ld, at["right.b"].addr, lane.proj.ld, st["S"], 1, m.dim ** -0.5,
                           ("delta", run))
        s_n = head_norm_stage(lane, p, [s_m, s_g], T, m, lane.gate, w.norm, 0, ("delta_norm", run))
        return lane.closing(p, s_n, lane.mix, w.o, T, m.heads * m.vdim, ("delta_o", run))


class Parallel:
    """Two mixers on one input, half the sum of their outputs, each normed: attention on the left, a gated delta rule on the
    right.  The norms and the sum are part of the residual stage behind the mixer (tile 66)."""

    BRANCH_SCALE = 0.5

    @staticmethod
    def check(i, m):
        GroupedAttention.check(i, m["left"])
        GatedDelta.check(i, m["right"])
        m["left"], m["right"] = types.SimpleNamespace(**m["left"]), types.SimpleNamespace(**m["right"])

    @staticmethod
    def place(W, w, m, g):
        w.stack = Stack(GatedDelta.blocks(g) + GroupedAttention.blocks(g))
        w.in_, w.left, w.right = W.mat(w.stack.rows), GroupedAttention.place(W, m.left, g), GatedDelta.place(W, m.right, g)
        w.branches = (w.right.out, w.left.out)   # in the order of `closing`'s outputs y, y2

    @staticmethod
    def state(cfg, m, rows, slots, page):
        return dict(GatedDelta.state(m.right, slots), **GroupedAttention.state(cfg, m.left, rows, page))

    @staticmethod
    def sizes(m, w):
        return dict(GatedDelta.sizes(m.right), **GroupedAttention.sizes(m.left), proj=w.stack.n, y2=1)

    @staticmethod
    def prepare(lane, layer, w, st):
        lane.weight_map(w.in_), lane.weight_map(w.left.o)
        GatedDelta.prepare(lane, layer.m.right, w.right, w.stack.at)
        GroupedAttention.prepare(lane, layer.m.left, st)

    @staticmethod
    def build(lane, p, l, run, b, prev):
        m, w, st = lane.cfg.layers[l].m, lane.w.layers[l], lane.kv.runs[run]
        s = lane.product(p, prev, lane.h, w.in_, lane.proj, b.T, w.stack.n, lane.cfg.hidden, ("parallel_in", run), out16=True)
        at = {name: lane.proj.view(col) for name, col in w.stack.at.items()}
        right, (parts0,) = GatedDelta.build(lane, p, m.right, w.right, st, at, run, b, s)
        left, (parts1,) = GroupedAttention.build(lane, p, m.left, w.left, st, at, run, b, s)
        return [right, left], (parts0, parts1)

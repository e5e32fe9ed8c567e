"""Layer-list decoders as fabric lane programs: the configuration names the mixer of every layer.  What differs between
designs otherwise is in DESIGNS: Sinotar (selective scan, latent attention, matrix memory; the residual a set of
hyper-connected streams; a span of layers may run several times in a row) and Teganex (gated linear attention, and
attention beside a gated delta rule: monoserve_b200/gated_mixers.py; a plain residual normed before and after each
sublayer).

`LayerListLane` builds the chain of one batch on the fabric's tiles, one run of a layer after the other:

  streams (53: update of the streams by the sublayer before, the next sublayer's input, its norm), or
  residual (66: the same for the plain residual)
    selective scan:    in GEMM (32) -> conv + silu (54) -> x GEMM (K ranges) -> slab sum (62) -> dt GEMM -> scan (55; one
                       token: 65) -> o GEMM
    matrix memory:     q k v g GEMM, gates GEMM beside it -> memory (57; one token: 56) -> head norm (58) -> o GEMM
    latent attention:  q + latent GEMM -> latent norm, rotation, cache append (59) -> per head W_uk^T q GEMM ->
                       attention over the cached latents (63 on the tensor cores, 60 in 32-bit; 61) -> per head W_uv
                       GEMM -> o GEMM; for a whole prompt: keys and values GEMM -> attention (64) -> o GEMM
    gated linear:      q k v g and low-rank decay GEMM -> decay GEMM with the decay epilogue -> gated memory (68; one token: 69) -> head norm (58) -> o GEMM
    parallel:          one GEMM for both sides; left: norms and append (70) -> paged attention (33 - 35, 44; 71 in 32-bit) ->
                       head gate (72) -> o GEMM; right: conv (54), decay and gate GEMMs -> gated memory (68, 69) ->
                       head norm (58) -> o GEMM
  streams -> gate / up GEMM with the gated epilogue -> down GEMM
  ... -> final streams (gather) -> head GEMM (fp32) -> sample (43)

Residuals, norms, positions, gates, scores and recurrent state are 32-bit; GEMM operands are bf16.  With
cfg.f32 set every activation is fp32 and every product runs in 32-bit arithmetic (tile 51): the exact form of the same
programs, for checking.

State: `LayerListCache` holds, per layer run, pages of latents or of keys and values (addressed through the lane's block
table) and slot-indexed recurrent state.  A request that starts at position 0 finds the state of its slot ignored (the tiles take
it as zero), so slots and pages are handed on without clearing.
"""
import types

import numpy as np
import torch

from monoserve_b200 import _C
from monoserve_b200.checkpoint import checkpoint_files, safetensors_tensors
from monoserve_b200.fabric import Program, Tile, tile_array
from monoserve_b200.fabric.args import pack
from monoserve_b200.gated_mixers import GatedLinear, Parallel
from monoserve_b200.lane_base import (EPI_F32, EPI_GELU_MUL, EPI_SILU_MUL, EPI_STORE, HEIGHTS, K_GEMM, K_SAMPLE, SPLIT_PARTS,
                                      SPLIT_ROWS, LaneBase, _bm, _retarget, up)

K_PRODUCT, K_GATED, K_STREAMS, K_CONV, K_SCAN, K_MEMORY_STEP, K_MEMORY, K_SCAN_STEP = 51, 52, 53, 54, 55, 56, 57, 65
K_RESIDUAL = 66
K_HEAD_NORM, K_LATENT_KV, K_LATENT_ATTN, K_LATENT_MERGE, K_SUM, K_LATENT_MMA, K_LATENT_DIRECT = 58, 59, 60, 61, 62, 63, 64
MAX_STREAMS, MAX_TAPS, MAX_SCAN_STATE, MAX_MEMORY_DIM, MAX_LATENT_DIM = 8, 8, 128, 512, 1152
SCAN_CHANNELS, MEMORY_COLUMNS, STEP_CHANNELS = 32, 32, 512   # of one tile
WIDE_ROWS, WIDE_PARTS = 512, 4           # K ranges of the products that end a sublayer, up to this many rows
MAX_ATTN_PARTS, ATTN_ROUNDS = 32, 1
RING_BYTES, KEY_TILE = 216 * 1024, 128   # shared memory of a wide tile; keys per step of the tensor-core attention tiles
DIRECT_ROWS = 32                         # a prompt of at least this many tokens maps its keys and values out of the latents


# What a design fixes: its registry name, the mixers it has, what a norm weight is counted from, the feed-forward's
# activation, and its residual: "streams", or "normed" on both sides of a sublayer.
DESIGNS = {
    "Sinotar": types.SimpleNamespace(name="sinotar", mixers=("mamba1", "mlstm", "latent_attention"), norm_from=1, act="gelu",
                                     residual="streams"),
    "Teganex": types.SimpleNamespace(name="teganex", mixers=("gla", "parallel"), norm_from=0, act="silu", residual="normed"),
}


# ---------------------------------------------------------------------------------------------- configuration
def read_config(c, dtype="bfloat16"):
    """The model shape from a parsed config.json with a list of layers."""
    if dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {dtype}")
    design = DESIGNS[c.get("architecture", "Sinotar")]
    layers = []
    for i, e in enumerate(c["layers"]):
        kind, m, mlp = e["type"], dict(e["mixer"]), e.get("mlp")
        if kind not in design.mixers:
            raise NotImplementedError(f"layer {i}: mixer {kind}")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise NotImplementedError(f"layer {i}: feed-forward {mlp['kind']}")
        MIXERS[kind].check(i, m)
        layers.append(types.SimpleNamespace(kind=kind, m=types.SimpleNamespace(**m), ff=mlp["ff"] if mlp else 0))
    loop = c.get("loop")
    order = list(range(len(layers)))
    if loop:
        a, b = loop["start"], loop["stop"]
        order = order[:a] + order[a:b] * loop["times"] + order[b:]
    streams = c["streams"] if design.residual == "streams" else 1
    if not 1 <= streams <= MAX_STREAMS:
        raise NotImplementedError(f"{streams} residual streams (1 to {MAX_STREAMS})")
    return types.SimpleNamespace(model_type=design.name, design=design, hidden=c["width"], vocab=c["vocab"],
                                 eps=float(c["norm"]["eps"]), streams=streams, layers=layers, order=order,
                                 num_layers=len(layers), f32=dtype == "float32",
                                 embed_scale=float(c.get("embedding", {}).get("scale", 1.0)),
                                 logit_scale=float(c.get("logit_scale", 1.0)), max_positions=c.get("max_positions"))


def read_tensors(folder):
    """{name: CPU tensor} of a checkpoint folder."""
    return {name: t.clone() for path in checkpoint_files(folder) for name, t in safetensors_tensors(path)}


class Weights:
    """Device placement of one decoder's tensors ({name: tensor}, linear weights [out, in]): matrices in bf16 with rows
    padded to whole 64-element K steps, everything that enters 32-bit arithmetic in fp32.  Products that read the same
    input are stacked.  Layers that run several times are placed once."""

    def __init__(self, cfg, tensors):
        self.cfg = cfg
        t = tensors
        design = cfg.design
        self.embed = t["embed"].to(torch.bfloat16).contiguous().cuda()
        self.pos = t["pos"].to(torch.bfloat16).contiguous().cuda() if "pos" in t else None
        self.head = self.mat(t["head"])
        # the logits' scale goes with the row in front of the head product
        self.final_norm = self.f32((design.norm_from + t["final.norm"].float()) * cfg.logit_scale)
        self.ones = torch.ones(cfg.streams, device="cuda")
        self.layers = []
        for l, layer in enumerate(cfg.layers):
            g = lambda name: t[f"l{l}.{name}"]  # noqa: B023, E731
            norm = lambda name: self.f32(design.norm_from + g(name).float())  # noqa: B023, E731
            # in front of the sublayer, and behind it: (hc_out, hc_mix) of the streams, or the norm of its output
            after = (lambda i: [self.f32(g(f"hc{i}.{n}").float()) for n in ("in", "out", "mix")]) if design.residual == "streams" \
                else (lambda i: [None, norm(f"norm{i}b")])  # noqa: B023
            w = types.SimpleNamespace(norm1=norm("norm1"), hc1=after(1))
            MIXERS[layer.kind].place(self, w, layer.m, lambda name: g("mix." + name))
            if layer.ff:
                w.norm2, w.hc2 = norm("norm2"), after(2)
                w.gate_up = self.mat(torch.cat([g("mlp.gate"), g("mlp.up")]))
                w.down = self.mat(g("mlp.down"))
            self.layers.append(w)

    @staticmethod
    def f32(t):
        return t.float().contiguous().cuda()

    @staticmethod
    def mat(t):
        """bf16 [.., out, in padded to 64]."""
        k = t.shape[-1]
        return torch.nn.functional.pad(t.to(torch.bfloat16), (0, up(k, 64) - k)).contiguous().cuda()


class LayerListCache:
    """Cache and state of every layer run, shared by the lanes: `page` tokens per page of latents, or of keys and values
    (page 0 is the sink unused block-table entries point at), `slots` requests' recurrent state."""

    def __init__(self, cfg, n_pages, page_size=16, slots=8):
        self.n_pages, self.page, self.slots = n_pages, page_size, slots
        self.runs = [MIXERS[cfg.layers[l].kind].state(cfg, cfg.layers[l].m, n_pages * page_size, slots, page_size)
                     for l in cfg.order]


def latent_tile(m, page, tokens_per_request):
    """(tokens, heads, key-tile buffers) of a tensor-core attention tile (kind 63), or None where its operands do not fit
    the worker's shared memory or TMEM, or the page size does not divide a key tile (kind 60 then)."""
    chunks, blocks = -(-(m.kv_rank + m.rot_dim) // 64), -(-m.kv_rank // 128)
    if page % 8 or KEY_TILE % page:
        return None

    def room(cols, buffers):
        return cols * (chunks * 128 + 256) + buffers * chunks * KEY_TILE * 128 <= RING_BYTES and blocks * cols <= 448

    most = next((n for n in (64, 32, 16) if room(n, 1)), None)
    if most is None:
        return None
    heads = -(-m.heads // -(-m.heads // most))
    tokens = max(1, min(most // heads, tokens_per_request))
    cols = next(n for n in (16, 32, 64) if n >= tokens * heads)
    return tokens, heads, 2 if room(cols, 2) else 1


def direct_buffers(m):
    """Key-tile buffers of the whole-prompt attention tile (kind 64), or 0 where its operands do not fit."""
    if any(v % 8 for v in (m.dim, m.rot_dim, m.vdim, m.kv_rank)) or m.vdim > 256:
        return 0
    nq, ne, room = -(-m.dim // 64) + -(-m.rot_dim // 64), -(-m.vdim // 64), RING_BYTES // (KEY_TILE * 128)
    return next((b for b in (2, 1) if nq * (1 + b) + ne + 2 <= room), 0)


# ---------------------------------------------------------------------------------------------- mixers
class SelectiveScan:
    """x, z = W_in h; x through a causal convolution per channel and silu; dt, B, C from x;
    S <- exp(dt A) S + dt x B, y = S C + D x, y silu(z), W_o."""

    @staticmethod
    def check(i, m):
        if m["state"] > MAX_SCAN_STATE or not 1 <= m["conv"] <= MAX_TAPS:
            raise NotImplementedError(f"layer {i}: state {m['state']} (to {MAX_SCAN_STATE}), {m['conv']} taps (to {MAX_TAPS})")

    @staticmethod
    def place(W, w, m, g):
        w.in_, w.x, w.dt, w.o = W.mat(g("in")), W.mat(g("x")), W.mat(g("dt")), W.mat(g("o"))
        w.conv, w.conv_b, w.dt_b, w.D = W.f32(g("conv")), W.f32(g("conv.b")), W.f32(g("dt.b")), W.f32(g("D"))
        w.A = W.f32(-torch.exp(g("A_log").float()))

    @staticmethod
    def state(cfg, m, rows, slots, page):
        return dict(state=torch.zeros(slots, m.inner, m.state, device="cuda"),
                    tail=torch.zeros(slots, max(1, m.conv - 1), m.inner, device="cuda"))

    @staticmethod
    def sizes(m, w):
        return dict(proj=2 * m.inner, act=m.inner, mix=m.inner, small=m.dt_rank + 2 * m.state, dt=m.inner, dt_in=m.dt_rank)

    @staticmethod
    def prepare(lane, layer, w, st):
        m = layer.m
        for t in (w.in_, w.x, w.dt, w.o):
            lane.weight_map(t)
        lane.act.maps(m.inner), lane.dt_in.maps(m.dt_rank), lane.mix.maps(m.inner)

    @staticmethod
    def build(lane, p, l, run, b, prev):
        m, w, st, T = lane.cfg.layers[l].m, lane.w.layers[l], lane.kv.runs[run], b.T
        f32, R = int(lane.cfg.f32), m.dt_rank + 2 * m.state
        s = lane.product(p, prev, lane.h, w.in_, lane.proj, T, 2 * m.inner, lane.cfg.hidden, ("scan_in", run), out16=True)
        conv = lane._dev("ConvArgs", x=lane.proj.addr, tail=st["tail"], w=w.conv, bias=w.conv_b, out=lane.act.addr,
                         tok_pos=lane.tok_pos, ld_x=lane.proj.ld, ld_out=lane.act.ld, channels=m.inner, taps=m.conv, f32=f32)
        s_conv = p.stage(_retarget(b.conv_tiles(m.inner), a0=conv.data_ptr()), label=("conv", run))
        p.after(s, s_conv)
        if f32:
            s_x = lane.product(p, s_conv, lane.act, w.x, lane.small, T, R, m.inner, ("scan_x", run))
            dt_in = lane.small
        else:
            parts = lane.split_parts(T, m.inner)
            s_x = lane.product(p, s_conv, lane.act, w.x, lane.slabs, T, R, m.inner, ("scan_x", run), parts=parts, ld_out=R)
            sm = lane._dev("SumArgs", out32=lane.small.addr, out16=lane.dt_in.addr, cols=R, parts=parts,
                           part_rows=lane.slab_rows(T), ld_in=R, ld_32=lane.small.ld, ld_16=lane.dt_in.ld, c16=m.dt_rank,
                           **{"in": lane.slabs.addr})
            s_sum = p.stage(lane._rows(K_SUM, sm, T, lane._per(T)), label=("scan_sum", run))
            p.after(s_x, s_sum)
            s_x, dt_in = s_sum, lane.dt_in
        s_dt = lane.product(p, s_x, dt_in, w.dt, lane.dt, T, m.inner, m.dt_rank, ("scan_dt", run))
        es = lane.proj.es
        sc = lane._dev("ScanArgs", x=lane.act.addr, z=lane.proj.addr + m.inner * es, dt=lane.dt.addr, dt_bias=w.dt_b,
                       b=lane.small.addr + 4 * m.dt_rank, c=lane.small.addr + 4 * (m.dt_rank + m.state), A=w.A, D=w.D,
                       state=st["state"], tail=st["tail"], x_in=lane.proj.addr, y=lane.mix.addr, tok_pos=lane.tok_pos,
                       ld_x=lane.act.ld, ld_z=lane.proj.ld, ld_dt=lane.dt.ld, ld_bc=lane.small.ld, ld_y=lane.mix.ld,
                       channels=m.inner, n=m.state, taps=m.conv, f32=f32)
        s_sc = p.stage(_retarget(b.scan_tiles(m.inner), a0=sc.data_ptr()), label=("scan", run))
        p.after(s_dt, s_sc)
        return lane.closing(p, s_sc, lane.mix, w.o, T, m.inner, ("scan_o", run))


class MatrixMemory:
    """q, k, v, g from h; log gates i = cap tanh((W_i h + b) / cap), f = logsigmoid(cap tanh(..)); per head
    S <- e^(f + m' - m) S + e^(i - m) k v^T with the running maximum m, read by q over max(|n q|, e^-m); head norm, gate."""

    @staticmethod
    def check(i, m):
        if m["dim"] > MAX_MEMORY_DIM:
            raise NotImplementedError(f"layer {i}: memory of {m['dim']} key dimensions (to {MAX_MEMORY_DIM})")

    @staticmethod
    def place(W, w, m, g):
        w.qkvg, w.o = W.mat(torch.cat([g(n) for n in "qkvg"])), W.mat(g("o"))
        gates = W.mat(torch.cat([g("i"), g("f")]))
        w.gates = gates if W.cfg.f32 else torch.cat([gates] * 3, -1).contiguous()   # one copy per part of a split row
        w.gate_b, w.norm = W.f32(torch.cat([g("i.b"), g("f.b")])), W.f32(g("norm"))

    @staticmethod
    def state(cfg, m, rows, slots, page):
        return dict(S=torch.zeros(slots, m.heads, m.vdim + 1, up(m.dim, 4), device="cuda"),
                    m=torch.zeros(slots, m.heads, up(m.vdim + 1, MEMORY_COLUMNS) // MEMORY_COLUMNS, device="cuda"))

    @staticmethod
    def sizes(m, w):
        return dict(proj=2 * m.heads * (m.dim + m.vdim), mix=m.heads * m.vdim, small=2 * m.heads, raw=m.heads * up(m.vdim + 1, 4),
                    split=1)

    @staticmethod
    def prepare(lane, layer, w, st):
        lane.weight_map(w.qkvg), lane.weight_map(w.gates), lane.weight_map(w.o)
        lane.h.maps(3 * lane.split), lane.mix.maps(layer.m.heads * layer.m.vdim)

    @staticmethod
    def build(lane, p, l, run, b, prev):
        m, w, st, T = lane.cfg.layers[l].m, lane.w.layers[l], lane.kv.runs[run], b.T
        f32, H, d, e, es = int(lane.cfg.f32), m.heads, m.dim, m.vdim, lane.proj.es
        s = lane.product(p, prev, lane.h, w.qkvg, lane.proj, T, 2 * H * (d + e), lane.cfg.hidden, ("memory_in", run), out16=True)
        # the gates enter the recurrence: their projection takes the whole 32-bit row, as three bf16 parts on the tensor cores
        k = lane.cfg.hidden if f32 else 3 * up(lane.cfg.hidden, 64)
        parts = 1 if f32 else lane.split_parts(T, k)
        raw, ld = (lane.slabs, 2 * H) if parts > 1 else (lane.small, lane.small.ld)
        s_g = lane.product(p, prev, lane.h, w.gates, raw, T, 2 * H, k, ("memory_gates", run), parts=parts, ld_out=ld)
        at = lane.proj.addr
        mem = lane._dev("MemoryArgs", q=at, k=at + es * H * d, v=at + es * 2 * H * d, gates=raw.addr,
                        gate_parts=parts, gate_rows=lane.slab_rows(T), gate_bias=w.gate_b, state=st["S"], m=st["m"], out=lane.raw.addr, tok_pos=lane.tok_pos,
                        ld_qkv=lane.proj.ld, ld_gates=ld, heads=H, d=d, e=e, f32=f32, q_scale=d ** -0.5, cap=m.gate_cap)
        s_m = p.stage(_retarget(b.memory_tiles(H, e), a0=mem.data_ptr()), label=("memory", run))
        p.after(s, s_m)
        p.after(s_g, s_m)
        nrm = lane._dev("HeadNormArgs", o=lane.raw.addr, g=at + es * H * (2 * d + e), w=w.norm, out=lane.mix.addr, heads=H,
                        e=e, ld_g=lane.proj.ld, ld_out=lane.mix.ld, f32=f32, eps=lane.cfg.eps, divide=1, w_head=e)
        s_n = p.stage(lane._rows(K_HEAD_NORM, nrm, T * H, lane.items_per(T * H)), label=("head_norm", run))
        p.after(s_m, s_n)
        return lane.closing(p, s_n, lane.mix, w.o, T, H * e, ("memory_o", run))


class LatentAttention:
    """Causal attention whose keys and values are linear maps of a cached latent (plus one rotated key part shared by
    the heads), in the absorbed form: W_uk^T q meets the latents themselves, W_uv maps their weighted sum."""

    @staticmethod
    def check(i, m):
        if m["kv_rank"] + m["rot_dim"] > MAX_LATENT_DIM:
            raise NotImplementedError(f"layer {i}: latent of {m['kv_rank']} + {m['rot_dim']} columns (to {MAX_LATENT_DIM})")
        if m["rot"]["dims"] != m["rot_dim"] or m["rot_dim"] % 2:
            raise NotImplementedError(f"layer {i}: rotation of {m['rot']['dims']} of {m['rot_dim']} columns")

    @staticmethod
    def place(W, w, m, g):
        w.qkv, w.o, w.c_norm = W.mat(torch.cat([g("q"), g("dkv")])), W.mat(g("o")), W.f32(g("dkv.norm"))
        w.ukv = W.mat(torch.cat([g("uk"), g("uv")]))
        w.uk = W.mat(g("uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2))    # [head][latent][dim]
        w.uv = W.mat(g("uv").view(m.heads, m.vdim, m.kv_rank))                   # [head][value][latent]

    @staticmethod
    def state(cfg, m, rows, slots, page):
        return dict(cache=torch.zeros(rows, up(m.kv_rank + m.rot_dim, 64), device="cuda",
                                      dtype=torch.float32 if cfg.f32 else torch.bfloat16))

    @staticmethod
    def sizes(m, w):
        return dict(qc=m.heads * (m.dim + m.rot_dim) + m.kv_rank + m.rot_dim, mix=m.heads * m.vdim,
                    kvb=m.heads * (m.dim + m.vdim), c_rows=m.kv_rank + m.rot_dim, q_un=(m.heads, m.dim), q_all=(m.heads, m.kv_rank + m.rot_dim), o_lat=(m.heads, m.kv_rank),
                    ws=(m.heads, m.kv_rank))

    @staticmethod
    def prepare(lane, layer, w, st):
        m = layer.m
        for t in (w.qkv, w.uk, w.uv, w.ukv, w.o):
            lane.weight_map(t)
        lane.mix.maps(m.heads * m.vdim)
        lane.head_maps(lane.q_un.addr, up(m.dim, 64), m.dim, m.heads)
        lane.head_maps(lane.o_lat.addr, up(m.kv_rank, 64), m.kv_rank, m.heads)
        lane.c_rows.maps(m.kv_rank)
        if direct_buffers(m):
            lane.direct_maps(m)
        for n in range(1, 65):   # a program's tile shape follows its longest request
            shape = latent_tile(m, lane.kv.page, n)
            if shape:
                lane.q_map(m, *shape[:2])
        if latent_tile(m, lane.kv.page, 1):
            lane.kv_map(m, st["cache"])

    @staticmethod
    def build(lane, p, l, run, b, prev):
        m, w, st, T = lane.cfg.layers[l].m, lane.w.layers[l], lane.kv.runs[run], b.T
        f32, H, d, r, c = int(lane.cfg.f32), m.heads, m.dim, m.rot_dim, m.kv_rank
        buffers = 0 if f32 else direct_buffers(m)
        whole, rest = b.split() if buffers else ([], b)
        s = lane.product(p, prev, lane.h, w.qkv, lane.qc, T, H * (d + r) + c + r, lane.cfg.hidden, ("latent_in", run))
        ld_q = up(c + r, 8)
        copy = dict(rows=lane.c_rows.addr, ld_rows=lane.c_rows.ld) if whole else {}
        kv = lane._dev("LatentArgs", qc=lane.qc.addr, c_norm=w.c_norm, q_un=lane.q_un.addr, q_all=lane.q_all.addr,
                       cache=st["cache"], tok_pos=lane.tok_pos, tok_slot=lane.tok_slot, cos_sin=lane.cos_sin(m.rot["base"], r),
                       ld_qc=lane.qc.ld, heads=H, d=d, r=r, kv_rank=c, ld_un=up(d, 64), ld_q=ld_q, rows_max=lane.T,
                       ld_cache=st["cache"].shape[1], max_pos=lane.max_pos, f32=f32, eps=lane.cfg.eps, **copy)
        s_kv = p.stage(lane._rows(K_LATENT_KV, kv, T, lane._per(T)), label=("latent_kv", run))
        p.after(s, s_kv)
        ends = []
        if whole:
            ends.append(LatentAttention.direct(lane, p, m, w, whole, buffers, T, run, s_kv))
        if rest.requests:
            ends.append(LatentAttention.absorbed(lane, p, m, w, st["cache"], rest, run, s_kv))
        return lane.closing(p, ends, lane.mix, w.o, T, H * m.vdim, ("latent_o", run))

    @staticmethod
    def direct(lane, p, m, w, requests, buffers, T, run, prev):
        """Whole prompts: keys and values of the prompt's own rows, then attention straight into `mix`."""
        H, d, r, e, c = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        s = lane.product(p, prev, lane.c_rows, w.ukv, lane.kvb, T, H * (d + e), c, ("latent_expand", run), out16=True)
        q_map, qr_map, kv_map, kr_map = lane.direct_maps(m)
        at = lane._dev("LatentDirectArgs", q_map=q_map, qr_map=qr_map, kv_map=kv_map, kr_map=kr_map, out=lane.mix.addr, d=d, r=r,
                       e=e, heads=H, rows_max=lane.T, ld_out=lane.mix.ld, buffers=buffers, scale=m.scale)
        blocks = sorted(((q0, row0, n) for row0, n, _ in requests for q0 in range(0, n, 128)), reverse=True)   # longest first
        q0, row0, n = (np.array(v)[:, None] for v in zip(*blocks))
        s_at = p.stage(tile_array(K_LATENT_DIRECT, i0=row0, i1=n, i2=q0, i3=np.arange(H)[None], a0=at.data_ptr()),
                       label=("latent_attn", run))
        p.after(s, s_at)
        return s_at

    @staticmethod
    def absorbed(lane, p, m, w, cache, b, run, prev):
        """Rows that attend to cached latents: W_uk^T q, attention over the latents themselves, W_uv."""
        f32, H, d, r, c = int(lane.cfg.f32), m.heads, m.dim, m.rot_dim, m.kv_rank
        ld_q, ld_o, spans = up(c + r, 8), up(c, 64), b.spans()
        s = lane.head_product(p, prev, lane.q_un.addr, up(d, 64), w.uk, lane.q_all.addr, ld_q, lane.T * ld_q, spans, c, d,
                              ("latent_q", run))
        shape = None if f32 else latent_tile(m, lane.kv.page, max(n for _, n, _ in b.requests))
        fields = dict(q=lane.q_all.addr, cache=cache, block_table=lane.bt, out=lane.o_lat.addr, ws_o=lane.ws.data_ptr(),
                      ws_ml=lane.ws_ml.data_ptr(), tok_pos=lane.tok_pos, ld_q=ld_q, heads=H, kv_rank=c, r=r,
                      ld_cache=cache.shape[1], page=lane.kv.page, bt_stride=lane.bt_stride, rows_max=lane.T, ld_out=ld_o,
                      f32=f32, scale=m.scale)
        if shape:
            tokens, heads, buffers = shape
            blocks = sum(-(-n // tokens) for _, n, _ in b.requests) * -(-H // heads)
            parts = lane.attn_parts(H, blocks)
            fields.update(q_map=lane.q_map(m, tokens, heads), kv_map=lane.kv_map(m, cache), tokens=tokens, group=heads,
                          buffers=buffers)
            tiles = b.latent_tiles(H, tokens, heads, parts)
        else:
            parts = lane.attn_parts(H, b.T * -(-H // 4))
            tiles = b.attn_tiles(H, parts)
        at = lane._dev("LatentAttnArgs", **fields)
        s_at = p.stage(_retarget(tiles, a0=at.data_ptr()), label=("latent_attn", run))
        p.after(s, s_at)
        if parts > 1:
            s_mg = p.stage(_retarget(b.item_tiles(K_LATENT_MERGE, H, i2=parts), a0=at.data_ptr()), label=("latent_merge", run))
            p.after(s_at, s_mg)
            s_at = s_mg
        return lane.head_product(p, s_at, lane.o_lat.addr, ld_o, w.uv, lane.mix.addr, lane.mix.ld, m.vdim, spans, m.vdim, c,
                                 ("latent_v", run))


MIXERS = {"mamba1": SelectiveScan, "mlstm": MatrixMemory, "latent_attention": LatentAttention, "gla": GatedLinear,
          "parallel": Parallel}


# ---------------------------------------------------------------------------------------------- the lane
class _Buf:
    """An activation buffer [rows][ld] and its tensor maps (bf16 operands of a GEMM)."""

    def __init__(self, lane, rows, cols, dtype):
        self.ld = up(cols, 64)
        self.t = torch.zeros(rows, self.ld, dtype=dtype, device="cuda")
        self.addr, self.es = self.t.data_ptr(), self.t.element_size()
        self.lane, self.rows, self._maps, self._views = lane, rows, {}, {}

    def data_ptr(self):
        return self.addr

    def view(self, col):
        """The buffer from column `col` on."""
        if col not in self._views:
            v = self._views[col] = object.__new__(_Buf)
            v.ld, v.t, v.addr, v.es, v.lane, v.rows, v._maps, v._views = \
                self.ld, None, self.addr + col * self.es, self.es, self.lane, self.rows, {}, {}
        return self._views[col]

    def maps(self, k):
        """Maps of the first k columns (zero beyond them)."""
        if k not in self._maps:
            self._maps[k] = [self.lane.fab.tensor_map(self.addr, [k, self.rows], [self.ld * 2], [64, bm]) for bm in HEIGHTS]
        return self._maps[k]


class _Batch:
    """The rows of one program: requests [(first row, rows, slot)], and the tile lists that depend on them only (made
    once per program and re-addressed per layer).  pos0: the requests' first positions, None for a decode step."""

    def __init__(self, lane, requests, pos0=None):
        self.lane, self.requests, self.pos0 = lane, requests, pos0
        self.T = sum(n for _, n, _ in requests)
        self.first, self.plans = None, []   # the program's first stage; plan tiles to be given their dynamic region
        self._made = {}

    def split(self):
        """(requests that bring a whole prompt from its start, a _Batch of the others)."""
        def make():
            whole = [i for i, (_, n, _) in enumerate(self.requests) if self.pos0 and self.pos0[i] == 0 and n >= DIRECT_ROWS]
            return [self.requests[i] for i in whole], _Batch(self.lane, [q for i, q in enumerate(self.requests) if i not in whole])
        return self._once("split", make)

    def spans(self):
        """The batch's rows as (first, rows), requests that lie side by side together."""
        out = []
        for row0, n, _ in self.requests:
            if out and sum(out[-1]) == row0:
                out[-1] = (out[-1][0], out[-1][1] + n)
            else:
                out.append((row0, n))
        return out

    def item_tiles(self, kind, per_row, **ops):
        """Item-wise tiles over the batch's rows, items row * per_row + j."""
        def make():
            per = self.lane.items_per(self.T * per_row)
            spans = [(row0 * per_row + i, min(per, n * per_row - i)) for row0, n in self.spans() for i in range(0, n * per_row, per)]
            first, count = (np.array(v) for v in zip(*spans))
            return tile_array(kind, i0=first, i1=count, **ops)
        return self._once((kind, per_row, tuple(ops.items())), make)

    def _once(self, key, make):
        if key not in self._made:
            self._made[key] = make()
        return self._made[key]

    def conv_tiles(self, channels):
        rows_per, ch_per = 32, 1024

        def make():
            out = []
            for row0, n, slot in self.requests:
                r, c = np.meshgrid(np.arange(0, n, rows_per), np.arange(0, channels, ch_per), indexing="ij")
                out.append(tile_array(K_CONV, i0=row0, i1=row0 + r,
                                      i2=np.minimum(rows_per, n - r) | (np.minimum(ch_per, channels - c) << 16), i3=slot, a1=c, a2=n))
            return np.concatenate(out)
        return self._once(("conv", channels), make)

    def scan_tiles(self, channels):
        """Portions: a tile per block of channels, the longest first; single tokens: wider blocks of one row each."""
        def make():
            out = [tile_array(K_SCAN, i0=row0, i1=n, i2=np.arange(0, channels, SCAN_CHANNELS), i3=slot)
                   for row0, n, slot in sorted(self.requests, key=lambda q: -q[1]) if n > 1]
            ones = [(row0, slot) for row0, n, slot in self.requests if n == 1]
            if ones:
                row, slot = (np.array(v)[:, None] for v in zip(*ones))
                c = np.arange(0, channels, STEP_CHANNELS)[None]
                out.append(tile_array(K_SCAN_STEP, i0=row, i1=np.minimum(STEP_CHANNELS, channels - c), i2=c, i3=slot))
            return np.concatenate(out)
        return self._once(("scan", channels), make)

    def memory_tiles(self, heads, e):
        """Portions: a tile per head and block of columns; single tokens: as many column blocks in a tile as leave every
        worker one."""
        def make():
            blocks = -(-(e + 1) // MEMORY_COLUMNS)
            h, c = np.meshgrid(np.arange(heads), np.arange(blocks), indexing="ij")
            out = [tile_array(K_MEMORY, i0=row0, i1=n, i2=h | (c << 16), i3=slot)
                   for row0, n, slot in sorted(self.requests, key=lambda q: -q[1]) if n > 1]
            ones = [(row0, slot) for row0, n, slot in self.requests if n == 1]
            if ones:
                row, slot = (np.array(v)[:, None, None] for v in zip(*ones))
                per = min(128, -(-blocks // min(blocks, max(1, self.lane.fab.num_workers // (len(ones) * heads)))))
                h, c = np.arange(heads)[None, :, None], np.arange(0, blocks, per)[None, None, :]
                out.append(tile_array(K_MEMORY_STEP, i0=row, i1=np.minimum(per, blocks - c), i2=h | (c << 16), i3=slot))
            return np.concatenate(out)
        return self._once(("memory", heads, e), make)

    def attn_tiles(self, heads, parts, kind=K_LATENT_ATTN):
        """One tile per row, group of heads and part, the rows that see most keys first."""
        per = 4 if parts > 1 or self.T * -(-heads // 4) <= 4 * self.lane.fab.num_workers else heads

        def make():
            rows = np.concatenate([np.arange(row0 + n - 1, row0 - 1, -1) for row0, n, _ in self.requests])
            slots = np.concatenate([np.full(n, slot) for _, n, slot in self.requests])
            h = np.arange(0, heads, per)
            return tile_array(kind, i0=rows[:, None, None], i1=(h | (np.minimum(per, heads - h) << 16))[None, :, None],
                              i2=np.arange(parts)[None, None, :], i3=parts, a1=slots[:, None, None])
        return self._once(("attn", heads, parts, kind), make)

    def latent_tiles(self, heads, tokens, group, parts):
        """One tile per block of `tokens` rows of a request, group of heads and part, the blocks that see most keys first
        (as far as the rows' order in their requests tells)."""
        def make():
            first = np.concatenate([row0 + np.arange(0, n, tokens) for row0, n, _ in self.requests])
            count = np.concatenate([np.minimum(tokens, n - np.arange(0, n, tokens)) for _, n, _ in self.requests])
            place = np.concatenate([np.arange(0, n, tokens) for _, n, _ in self.requests])
            slots = np.concatenate([np.full(-(-n // tokens), slot) for _, n, slot in self.requests])
            order = np.argsort(-place, kind="stable")
            r, n, s = (v[order][:, None, None] for v in (first, count, slots))
            h = np.arange(0, heads, group)[None, :, None]
            return tile_array(K_LATENT_MMA, i0=r, i1=n | (h << 16), i2=np.arange(parts)[None, None, :], i3=parts, a1=s)
        return self._once(("latent", heads, tokens, group, parts), make)


class LayerListLane(LaneBase):
    """One lane of the fabric running a layer-list decoder; the interface of ModelLane."""

    program = Program   # what programs are built with

    def __init__(self, fab, lane_id, cfg, weights, kv, max_tokens, max_slots, bt_stride, logit_rows=None, requests=None,
                 keep_residual=False):
        """keep_residual: every program also stores the sum of the streams after each layer run (`residual`)."""
        self.fab, self.lane_id, self.cfg, self.w, self.kv = fab, lane_id, cfg, weights, kv
        assert max_slots <= kv.slots, "the cache holds recurrent state for fewer slots"
        self.T, self.S, self.bt_stride = max_tokens, max_slots, bt_stride
        self.logit_rows = logit_rows or max(max_tokens, max_slots)
        T, H = max_tokens, cfg.hidden
        act, f32 = torch.float32 if cfg.f32 else torch.bfloat16, torch.float32
        z = lambda *shape, dt=torch.float32: torch.zeros(*shape, dtype=dt, device="cuda")  # noqa: E731
        sizes = {}
        for layer, lw in zip(cfg.layers, weights.layers):
            for name, v in MIXERS[layer.kind].sizes(layer.m, lw).items():
                if isinstance(v, tuple):   # per head: the largest block of heads x padded columns
                    sizes[name] = max(sizes.get(name, 0), v[0] * up(v[1], 64))
                else:
                    sizes[name] = max(sizes.get(name, 0), v)
        self.xs = z(T, cfg.streams, H)   # or the plain residual [T][H]
        # a row of h, and behind it what its bf16 rounding has left, for products that take the whole 32-bit row
        self.split = up(H, 64) if "split" in sizes and not cfg.f32 else 0
        self.h = _Buf(self, T, 3 * self.split or H, act)
        ff = max([layer.ff for layer in cfg.layers] + [0])
        self.hd = _Buf(self, T, ff, act) if ff else None
        self.gu = _Buf(self, T, 2 * ff, f32) if ff and cfg.f32 else None
        for name, dt in (("proj", act), ("act", act), ("mix", act), ("dt_in", act), ("mix2", act), ("gate", act), ("small", f32),
                         ("dt", f32), ("qc", f32), ("decay", f32), ("raw", f32)) + (() if cfg.f32 else (("kvb", act), ("c_rows", act))):
            setattr(self, name, _Buf(self, T, sizes[name], dt) if name in sizes else None)
        for name in ("q_un", "q_all", "o_lat", "gq", "go"):   # [head][T][columns] or [T][head][columns]: addressed by the layer's own strides
            if name in sizes:
                buf = types.SimpleNamespace(t=z(T * sizes[name], dt=act))
                buf.addr = buf.t.data_ptr()
                setattr(self, name, buf)
        # fp32 slabs of the K-split products: y of a sublayer, and the scan's x projection
        self.rows_slab = max(SPLIT_PARTS * SPLIT_ROWS, WIDE_PARTS * min(WIDE_ROWS, up(T, 64)), T)
        self.y = types.SimpleNamespace(t=z(self.rows_slab, H))
        self.y.addr = self.y.t.data_ptr()
        if "y2" in sizes:   # the second of two mixers side by side
            self.y2 = types.SimpleNamespace(t=z(self.rows_slab, H))
            self.y2.addr = self.y2.t.data_ptr()
        if "small" in sizes:
            self.slabs = types.SimpleNamespace(t=z(self.rows_slab * sizes["small"]))
            self.slabs.addr = self.slabs.t.data_ptr()
        if "ws" in sizes:
            self.ws_rows = max(min(T, SPLIT_ROWS), 1) * MAX_ATTN_PARTS * max(x.m.heads for x in cfg.layers if x.kind == "latent_attention")
            self.ws, self.ws_ml = z(self.ws_rows * max(x.m.kv_rank for x in cfg.layers if x.kind == "latent_attention")), z(self.ws_rows, 2)
        self.xlast, self.logits = _Buf(self, self.logit_rows, H, act), z(self.logit_rows, cfg.vocab)
        self.residual = z(len(cfg.order), T, H) if keep_residual else None
        self._request_state(T, self.S, requests)
        self.max_pos = bt_stride * kv.page
        self._cos_sin, self._wmaps, self._hmaps, self.attn_blocks = {}, {}, {}, {}
        for layer in cfg.layers:
            if layer.kind == "latent_attention":
                self.cos_sin(layer.m.rot["base"], layer.m.rot_dim)
        self._build_state((48 << 10) * (len(cfg.order) + 2))
        self.sample_args, self.step_args = self._sample_block(cfg.vocab), self._step_block()
        self._prepare()

    def _prepare(self):
        """Make every tensor map a program can name now: none may be made while the fabric is resident."""
        if self.cfg.f32:
            return
        cfg, w = self.cfg, self.w
        wm = self.weight_map
        wm(w.head)
        self.h.maps(cfg.hidden)
        self.xlast.maps(cfg.hidden)
        for layer, lw in zip(cfg.layers, w.layers):
            if layer.ff:
                wm(lw.gate_up), wm(lw.down), self.hd.maps(layer.ff)
        for l, state in zip(cfg.order, self.kv.runs):
            layer, lw = cfg.layers[l], w.layers[l]
            MIXERS[layer.kind].prepare(self, layer, lw, state)

    def cos_sin(self, base, r):
        """fp32 [max_pos][r / 2][cos, sin] of the angles pos * base^(-2 i / r)."""
        if (base, r) not in self._cos_sin:
            f = float(base) ** (-2.0 * torch.arange(r // 2, dtype=torch.float64) / r)
            a = torch.arange(self.max_pos, dtype=torch.float64)[:, None] * f[None]
            self._cos_sin[base, r] = torch.stack([a.cos(), a.sin()], -1).float().contiguous().cuda()
        return self._cos_sin[base, r]

    # ------------------------------------------------------------------ products
    def weight_map(self, t):
        if t.data_ptr() not in self._wmaps:
            self._wmaps[t.data_ptr()] = self._wmap(t)
        return self._wmaps[t.data_ptr()]

    def head_maps(self, addr, ld, k, heads):
        """Maps of the first k columns of a [head * T][ld] operand (zero beyond them)."""
        key = addr, ld, k, heads
        if key not in self._hmaps:
            self._hmaps[key] = [self.fab.tensor_map(addr, [k, heads * self.T], [ld * 2], [64, bm]) for bm in HEIGHTS]
        return self._hmaps[key]

    def split_parts(self, rows, k):
        """K ranges of a product that ends in fp32 slabs."""
        if rows > min(WIDE_ROWS, up(self.T, 64)):
            return 1
        return max(1, min(SPLIT_PARTS if rows <= SPLIT_ROWS else WIDE_PARTS, -(-k // 64) // 8))

    def slab_rows(self, rows):
        return SPLIT_ROWS if rows <= SPLIT_ROWS else min(WIDE_ROWS, up(self.T, 64)) if rows <= WIDE_ROWS else self.T

    def product(self, p, prev, x, w, out, rows, n, k, label, out16=False, parts=1, ld_out=None, epi=None, up_offset=0,
                bias=None, coef=None):
        """A stage out[rows][n] = x[rows][k] w[n][k]^T after `prev`.  out16: the output is of the activations' type,
        else fp32; parts > 1: that many fp32 slabs."""
        ld = ld_out or out.ld
        if self.cfg.f32:
            args = self._dev("ProductArgs", x=x.addr, w=w, out=out.addr, ld_x=x.ld, ld_w=w.shape[-1], ld_out=ld, K=k, N=n, f32=1)
            s = p.stage(_retarget(self._product_tiles(rows, n), a0=args.data_ptr()), label=label)
        elif parts > 1:
            s = self._gemm_split(p, self.weight_map(w), x.maps(k), rows, n, k, out.t, parts, label,
                                 slab_rows=self.slab_rows(rows))
        else:
            s = self._gemm(p, self.weight_map(w), x.maps(k), rows, n, k, out.t, ld,
                           epi if epi is not None else (EPI_STORE if out16 else EPI_F32), label, up_offset=up_offset,
                           bm=self.row_block(rows, n), bias=bias, coef=coef)
        for stage in prev if isinstance(prev, list) else [prev]:
            p.after(stage, s)
        return s

    def row_block(self, rows, n):
        """Row-block height of a GEMM: the largest that still gives most workers a tile (a narrow product over many rows
        takes lower blocks), at least 32 rows."""
        for bm in reversed(HEIGHTS):
            if bm <= _bm(rows) and -(-rows // bm) * -(-n // 128) * 4 >= 3 * self.fab.num_workers:
                return bm
        return min(32, _bm(rows))

    def _product_tiles(self, rows, n, row0=0):
        key = ("product", rows, n, row0)
        if key not in self._templates:
            r, c = np.meshgrid(np.arange(0, rows, 32), np.arange(0, n, 32), indexing="ij")
            self._templates[key] = tile_array(K_PRODUCT, i0=row0 + r, i1=np.minimum(32, rows - r), i2=c, i3=np.minimum(32, n - c))
        return self._templates[key]

    def head_product(self, p, prev, x_addr, ld_x, w, out_addr, ld_out, head_stride, spans, n, k, label):
        """Per head h and row span (first, rows): out[h * head_stride + row * ld_out ..n] = x[h * T + row][k] w[h][n][k]^T,
        activations' type out."""
        heads = w.shape[0]
        if self.cfg.f32:
            # tile 51 stores fp32, which is the activations' type here
            args = self._dev("ProductArgs", x=x_addr, w=w, out=out_addr, ld_x=ld_x, ld_w=w.shape[-1], ld_out=ld_out, K=k, N=n, f32=1)
            base = np.concatenate([self._product_tiles(rows, n, row0) for row0, rows in spans])
            tiles = np.tile(base, (heads, 1))
            h = np.repeat(np.arange(heads, dtype=np.uint64), len(base))
            tiles[:, 3] = args.data_ptr()
            tiles[:, 4] = h * np.uint64(4 * self.T * ld_x)
            tiles[:, 5] = h * np.uint64(2 * w.shape[1] * w.shape[2])
            tiles[:, 6] = h * np.uint64(4 * head_stride)
            s = p.stage(tiles, label=label)
        else:
            tiles = []
            for bm in sorted({_bm(rows) for _, rows in spans}):
                # the tile's activation rows are h * T + m and its output row is counted from there: the base makes up for it
                args = [self.arena.put(_C.gemm_args(out=(out_addr + 2 * (h * head_stride - h * self.T * ld_out)) % (1 << 64),
                                                    ld_out=ld_out, k_tiles=-(-k // 64), epi=EPI_STORE, bm=bm, n_limit=n)).data_ptr()
                        for h in range(heads)]
                m0, count = (np.array(v) for v in zip(*[(row0 + i, min(bm, rows - i)) for row0, rows in spans if _bm(rows) == bm
                                                        for i in range(0, rows, bm)]))
                h, m, n0 = np.meshgrid(np.arange(heads), np.arange(len(m0)), np.arange(0, n, 128), indexing="ij")
                tiles.append(tile_array(K_GEMM, i0=n0, i1=h * self.T + m0[m], i2=count[m], i3=h,
                                        a0=np.asarray(args, dtype=np.int64)[h], a1=self.weight_map(w),
                                        a2=self.head_maps(x_addr, ld_x, k, heads)[HEIGHTS.index(bm)]))
            tiles = np.concatenate(tiles)
            s = p.stage(tiles, label=label)
        p.after(prev, s)
        return s

    def closing(self, p, prev, x, w, rows, k, label, out=None):
        """The product that ends a sublayer: y (or `out`) as fp32 slabs for the streams or residual tile.  Returns (stage,
        (slabs,)); a sublayer of two mixers has a pair of each."""
        parts = 1 if self.cfg.f32 else self.split_parts(rows, k)
        s = self.product(p, prev, x, w, out or self.y, rows, self.cfg.hidden, k, label, parts=parts, ld_out=self.cfg.hidden)
        return s, (parts,)

    def items_per(self, items):
        """Items (one warp each) per tile of an item-wise stage: a multiple of four, about two rounds of tiles."""
        return max(4, up(-(-items // (2 * self.fab.num_workers)), 4))

    def q_map(self, m, tokens, heads):
        """The absorbed queries [head][T][columns], boxes of 64 columns x tokens x heads."""
        key = "q", m.kv_rank, m.rot_dim, m.heads, tokens, heads
        if key not in self._hmaps:
            ld = up(m.kv_rank + m.rot_dim, 8)
            self._hmaps[key] = self.fab.tensor_map(self.q_all.addr, [m.kv_rank + m.rot_dim, self.T, m.heads],
                                                   [ld * 2, self.T * ld * 2], [64, tokens, heads])
        return self._hmaps[key]

    def kv_map(self, m, cache):
        """A cache of latents, one box per page: groups of eight rows, their 64-column chunks side by side."""
        key = cache.data_ptr()
        if key not in self._hmaps:
            rows, ld = cache.shape
            chunks = -(-(m.kv_rank + m.rot_dim) // 64)
            self._hmaps[key] = self.fab.tensor_map(cache.data_ptr(), [64, 8, chunks, rows // 8], [ld * 2, 128, 16 * ld],
                                                   [64, 8, chunks, self.kv.page // 8])
        return self._hmaps[key]

    def attn_parts(self, heads, tiles):
        """Key ranges per row: as many as give every worker one tile (the split workspace is addressed by
        row, so it covers the rows of a small program only)."""
        want = min(MAX_ATTN_PARTS, ATTN_ROUNDS * self.fab.num_workers // tiles)
        return max(1, want) if self.rows_now <= SPLIT_ROWS else 1

    def direct_maps(self, m):
        """Operands of the whole-prompt attention tile: (q unrotated, q rotated, keys and values, rotated keys)."""
        key = "direct", m.dim, m.rot_dim, m.vdim, m.kv_rank, m.heads
        if key not in self._hmaps:
            box, H, T, ld_q = [64, KEY_TILE], m.heads, self.T, up(m.kv_rank + m.rot_dim, 8)
            tm = self.fab.tensor_map
            self._hmaps[key] = (tm(self.q_un.addr, [m.dim, H * T], [2 * up(m.dim, 64)], box),
                                tm(self.q_all.addr + 2 * m.kv_rank, [m.rot_dim, H * T], [2 * ld_q], box),
                                tm(self.kvb.addr, [H * (m.dim + m.vdim), T], [2 * self.kvb.ld], box),
                                tm(self.c_rows.addr + 2 * m.kv_rank, [m.rot_dim, T], [2 * self.c_rows.ld], box))
        return self._hmaps[key]

    # ------------------------------------------------------------------ programs
    def _between(self, p, rows, prev, sub, before, label, split=False, gather=False, step=False):
        """The stage between two sublayers: the residual takes the output of the one behind it, and the one ahead of it,
        `sub` = (hc_in, norm), gets its input.  `before` = (what of the layer's weights follows the sublayer, its slab
        counts, its branches' norms or None, run whose residual this completes or None), or None at the embedding."""
        cfg = self.cfg
        hc_in, norm = sub
        streams = cfg.design.residual == "streams"
        f = dict(w=norm, W=cfg.hidden, eps=cfg.eps)
        f.update(dict(xs=self.xs, hc_in=hc_in, streams=cfg.streams) if streams else dict(x=self.xs))
        if before is None:
            f.update(embed=self.w.embed, **({"step": self.step_args} if step else {"tokens": self.tokens}))
            if not streams:
                f.update(embed_scale=cfg.embed_scale, tok_pos=self.tok_pos, max_pos=self.max_pos)
                if self.w.pos is not None:
                    f.update(pos=self.w.pos, max_pos=self.w.pos.shape[0])
        else:
            after, parts, branches, run = before
            y_rows = self.slab_rows(rows)
            if streams:
                f.update(y=self.y.addr, hc_out=after[0], hc_mix=after[1], y_parts=parts[0], y_rows=y_rows)
            else:
                f.update(y0=self.y.addr, y0_parts=parts[0], y_rows=y_rows, post_w=after[0])
                if branches:
                    f.update(y1=self.y2.addr, y1_parts=parts[1], w0=branches[0], w1=branches[1],
                             branch_scale=Parallel.BRANCH_SCALE)
            if run is not None and self.residual is not None:
                f.update(sum_out=self.residual[run])
        if gather:
            f.update(gather=self.gather, ld_out=self.xlast.ld, **{"out32" if cfg.f32 else "out16": self.xlast.addr})
        elif cfg.f32:
            f.update(h32=self.h.addr, ld_h32=self.h.ld)
        else:
            f.update(h16=self.h.addr, ld_h16=self.h.ld)
            if split:
                f.update(split=self.split)
        args = self._dev("StreamArgs" if streams else "ResidualArgs", **f)
        s = p.stage(self._rows(K_STREAMS if streams else K_RESIDUAL, args, rows, self._per(rows)), label=label)
        if prev is not None:
            for stage in prev if isinstance(prev, list) else [prev]:
                p.after(stage, s)
        return s

    def _chain(self, p, b, step):
        """Every layer run; returns (first stage, the final stage of the residual)."""
        cfg, T = self.cfg, b.T
        self.rows_now = T
        name = "streams" if cfg.design.residual == "streams" else "residual"
        prev = before = None
        for run, l in enumerate(cfg.order):
            layer, w = cfg.layers[l], self.w.layers[l]
            prev = self._between(p, T, prev, (w.hc1[0], w.norm1), before, (name, run), split=layer.kind == "mlstm", step=step)
            b.first = prev if b.first is None else b.first
            prev, parts = MIXERS[layer.kind].build(self, p, l, run, b, prev)
            before = (w.hc1[1:], parts, getattr(w, "branches", None), None if layer.ff else run)
            if layer.ff:
                prev = self._between(p, T, prev, (w.hc2[0], w.norm2), before, (name + "_ff", run))
                if cfg.f32:
                    s = self.product(p, prev, self.h, w.gate_up, self.gu, T, 2 * layer.ff, cfg.hidden, ("ff_in", run))
                    g = self._dev("GatedArgs", out=self.hd.addr, ff=layer.ff, ld_in=self.gu.ld, ld_out=self.hd.ld,
                                  silu=int(cfg.design.act == "silu"), **{"in": self.gu.addr})
                    s_g = p.stage(self._rows(K_GATED, g, T, self._per(T)), label=("ff_act", run))
                    p.after(s, s_g)
                    s = s_g
                else:
                    s = self.product(p, prev, self.h, w.gate_up, self.hd, T, layer.ff, cfg.hidden, ("ff_in", run),
                                     epi=EPI_SILU_MUL if cfg.design.act == "silu" else EPI_GELU_MUL, up_offset=layer.ff)
                prev, parts = self.closing(p, s, self.hd, w.down, T, layer.ff, ("ff_out", run))
                before = (w.hc2[1:], parts, None, run)
        last = self._between(p, T, prev, (self.w.ones, self.w.final_norm), before, ("final", len(cfg.order)), gather=True)
        return b.first, last

    def _finish(self, p, b, prev, n_rows, sample_rows):
        if n_rows:
            s = self.product(p, prev, self.xlast, self.w.head, types.SimpleNamespace(t=self.logits, addr=self.logits.data_ptr(),
                                                                                     ld=self.cfg.vocab),
                             n_rows, self.cfg.vocab, self.cfg.hidden, ("head", -1))
            tiles = [Tile(K_SAMPLE, i=(row, slot), a=(self.sample_args.data_ptr(),)) for row, slot in sample_rows if row >= 0]
            if tiles:
                s_s = p.stage(tiles, label=("sample", -1))
                p.after(s, s_s)
        at = p.dynamic_first   # every static tile is counted: the plan tiles get their parts of the dynamic region
        for blob, fields, most in b.plans:
            p.reserve(most)
            self.arena.patch(blob, pack("AttnPlanArgs", dyn_first=at, dyn_cap=most, **fields))
            at += most
        self.rows_out = n_rows
        self.labels = p.labels()
        self.arena.flush()

    def build_prefill(self, batch, iterations=1, all_logits=False, want=None):
        """batch: [(slot, tokens, pos0)], a prompt or a portion of one each, pages in place.  Computes the rows, advances
        the requests' caches and states, and samples one next token per request, as ModelLane.build_prefill does.
        want: per request, the places among its tokens whose logits are kept instead (row by row in `logits`); then
        nothing is sampled."""
        self._reset_build()
        places = want if want is not None else [[len(toks) - 1] for _, toks, _ in batch]
        T, req_info, sample_rows = self._batch_rows(batch, places, all_logits)
        p = self.program()
        b = _Batch(self, [(row0, n, slot) for (row0, _, n, _), (slot, _, _) in zip(req_info, batch)], [q[2] for q in batch])
        first, last = self._chain(p, b, step=False)
        self._finish(p, b, last, T if all_logits else sum(len(v) for v in places), sample_rows if want is None else [])
        return p.upload(self.fab, first=first, iterations=iterations)

    def build_decode(self, slots, iterations=1, chunk_keys=0):
        """One decode step per iteration for the requests in `slots` (row r = slots[r])."""
        R = len(slots)
        assert 0 < R <= min(self.T, self.logit_rows)
        self._reset_build()
        self._put(self.row_req, slots)
        self._put(self.gather, np.arange(R))
        p = self.program()
        b = _Batch(self, [(r, 1, slot) for r, slot in enumerate(slots)])
        first, last = self._chain(p, b, step=True)
        self._finish(p, b, last, R, list(enumerate(slots)))
        return p.upload(self.fab, first=first, iterations=iterations)

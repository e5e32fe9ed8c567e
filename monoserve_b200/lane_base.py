"""What the lanes of every model family share: the operand arena of a program build, tensor maps, dense GEMM
stages, row-wise stages, the slot-indexed request state and the token rows of a prompt batch
(monoserve/runtime/lane.py:101-122,309-420 keeps these in its one lane class)."""
import struct

import numpy as np
import torch

from monoserve_b200 import _C
from monoserve_b200.fabric import tile_array
from monoserve_b200.fabric.args import pack

K_GEMM, K_SAMPLE = 32, 43
SPLIT_ROWS, SPLIT_PARTS = 64, 8   # a dense GEMM of at most SPLIT_ROWS rows may run as up to SPLIT_PARTS K ranges
EPI_STORE, EPI_SILU_MUL, EPI_F32, EPI_ROWS_F32, EPI_GELU_MUL, EPI_DECAY = 0, 1, 3, 5, 6, 7
GATED = (EPI_SILU_MUL, EPI_GELU_MUL)
HEIGHTS = [16, 32, 64, 128, 256]


def up(n, m):
    return -(-n // m) * m


def _block(name, **fields):
    return torch.frombuffer(bytearray(pack(name, **fields)), dtype=torch.uint8).cuda()


def _u64(values):
    return torch.tensor([int(v) for v in values], dtype=torch.int64).cuda()


class _Blob:
    """A piece of device memory by address (what `pack` and the tile builders need of a tensor)."""

    def __init__(self, addr, nbytes):
        self.addr, self.nbytes = addr, nbytes

    def data_ptr(self):
        return self.addr


class _Arena:
    """Device memory for the operand blocks of one program build, carved from one buffer that is
    allocated with the lane and filled through Fabric.write: a build then neither allocates device
    memory nor launches a kernel, both of which would wait for a resident fabric kernel."""

    def __init__(self, fab, nbytes):
        self.fab, self.buf, self.at = fab, torch.zeros(nbytes, dtype=torch.uint8, device="cuda"), 0
        self.host, self.flushed = bytearray(nbytes), 0   # the blocks of the current build; [flushed, at) not yet written

    def reset(self):
        self.at = self.flushed = 0

    def put(self, data):
        """Room for `data` in the arena; the bytes reach the device with the next flush()."""
        size = (len(data) + 255) & ~255
        if self.at + size > self.buf.numel():
            raise RuntimeError("monofab: the lane's operand arena is full")
        blob = _Blob(self.buf.data_ptr() + self.at, len(data))
        self.host[self.at:self.at + len(data)] = data
        self.at += size
        return blob

    def patch(self, blob, data):
        """Replace the contents of a block put earlier in this build."""
        at = blob.addr - self.buf.data_ptr()
        assert self.flushed <= at and at + len(data) <= self.at, "the block is not of the current build"
        self.host[at:at + len(data)] = data

    def flush(self):
        """One write of everything put since the last flush (a build has hundreds of blocks of 64 to 256 bytes)."""
        if self.at > self.flushed:
            self.fab.write(self.buf.data_ptr() + self.flushed, bytes(self.host[self.flushed:self.at]))
            self.flushed = self.at


def _bm(rows):
    """Row-block height of a dense GEMM over `rows` activation rows."""
    for h in HEIGHTS:
        if rows <= h:
            return h
    return HEIGHTS[-1]


def _retarget(template, a0=None, a1=None, a2=None, a4=None):
    """A copy of a tile array with other operand addresses.  The tiles of a stage depend on the layer only
    through the addresses they name, so a lane keeps one array per shape and re-addresses a copy per layer."""
    t = template.copy()
    for col, v in ((3, a0), (4, a1), (5, a2), (7, a4)):
        if v is not None:
            t[:, col] = v
    return t


def rope_table(theta, rot_dim, max_pos):
    """cos/sin fp32 [max_pos][rot_dim / 2][2], computed as the reference's oracle does
    (tests/test_fabric_model.py:35-42; the lane's host table: monoserve/runtime/lane.py:36-48)."""
    half = rot_dim // 2
    j = torch.arange(half, dtype=torch.float32)
    inv = 1.0 / torch.pow(torch.tensor(theta, dtype=torch.float32), 2 * j / rot_dim)
    ang = torch.arange(max_pos, dtype=torch.float32)[:, None] * inv[None]
    return torch.stack([ang.cos(), ang.sin()], -1).contiguous()


class Mat:
    """A weight matrix on the device: bf16, or e4m3 bytes with an fp32 scale per output row."""

    def __init__(self, data, scale=None):
        self.data, self.scale = data, scale
        self.fp8 = data.dtype == torch.uint8


class LaneBase:
    """One lane of the fabric.  A subclass sets fab, kv, logit_rows and T in its constructor and calls
    `_request_state` and `_build_state` there."""

    def _request_state(self, T, S, requests):
        """Token rows, and the slot-indexed request state: the lane's own, or a RequestTable's
        (monoserve/runtime/requests.py)."""
        z = lambda *shape, dt=torch.int32: torch.zeros(*shape, dtype=dt, device="cuda")  # noqa: E731
        self.tokens, self.tok_pos, self.tok_slot, self.gather = z(T), z(T), z(T), z(T)
        self.req_info = z(max(T, S), 4)
        self.row_req = z(max(T, S))
        if requests is not None:
            assert requests.slots >= S and requests.bt_stride == self.bt_stride
            self.bt, self.seq_len, self.last_token, self.steps = requests.bt, requests.seq_len, requests.last_token, requests.steps
            self.temperature, self.ring = requests.temperature, requests.ring
            self.host_tokens, self.host_steps = requests.host_tokens, requests.host_steps
        else:
            self.bt = z(S, self.bt_stride)
            self.seq_len, self.last_token, self.steps = z(S), z(S), z(S)
            self.temperature = z(S, dt=torch.float32)
            self.ring = 64
            self.host_tokens = torch.zeros(S, self.ring, dtype=torch.int32).pin_memory()
            self.host_steps = torch.zeros(S, dtype=torch.int64).pin_memory()

    def _build_state(self, arena_bytes):
        self._keep = []
        self.arena = _Arena(self.fab, arena_bytes)
        self._templates = {}   # tile arrays by shape, re-addressed per layer (_retarget)

    def _reset_build(self):
        self.arena.reset()   # the operand blocks of this lane's previous program: it must have ended
        if len(self._templates) > 256:   # shapes of many different batches: start over rather than grow
            self._templates.clear()

    def _sample_block(self, vocab):
        return _block("SampleArgs", logits=self.logits, temperature=self.temperature, last_token=self.last_token,
                      steps=self.steps, host_tokens=_C.host_device_pointer(self.host_tokens.data_ptr()),
                      host_steps=_C.host_device_pointer(self.host_steps.data_ptr()), seed=0x5eed, V=vocab, ring=self.ring)

    def _step_block(self):
        return _block("StepArgs", row_req=self.row_req, last_token=self.last_token, seq_len=self.seq_len,
                      block_table=self.bt, tok_pos=self.tok_pos, tok_slot=self.tok_slot, req_info=self.req_info,
                      bt_stride=self.bt_stride, page_size=self.kv.page)

    def _batch_rows(self, batch, want, all_rows=False):
        """The token rows of a prompt batch [(slot, tokens, pos0)] on the device: tokens, positions, cache slots and the
        logit row of every token row (gather; -1: none).  want: per request the places among its tokens whose logits are
        kept, in logit-row order (all_rows: every row).  Returns (rows, req_info, [(logit row of the request's last
        token or -1, slot)])."""
        page, stride = self.kv.page, self.bt.shape[1]
        tokens, pos, slots, req_info, gather, sample_rows = [], [], [], [], [], []
        row = kept = 0
        for i, (slot, toks, pos0) in enumerate(batch):
            n = len(toks)
            req_info.append((row, pos0, n, pos0 + n))
            # the request's row of the block table (read through the fabric: nothing may be launched beside it)
            pages = np.frombuffer(self.fab.read(self.bt.data_ptr() + 4 * slot * stride, 4 * stride), dtype=np.int32)
            ppos = pos0 + np.arange(n)
            tokens.append(np.asarray(toks, dtype=np.int32))
            pos.append(ppos.astype(np.int32))
            slots.append((pages[ppos // page].astype(np.int64) * page + ppos % page).astype(np.int32))
            places = np.arange(n) if all_rows else np.asarray(want[i], dtype=np.int64)
            g = np.full(n, -1, dtype=np.int32)
            g[places] = kept + np.arange(len(places), dtype=np.int32)
            gather.append(g)
            sample_rows.append((int(g[n - 1]), slot))
            row += n
            kept += len(places)
        assert 0 < row <= self.T and kept <= self.logit_rows
        self._put(self.tokens, np.concatenate(tokens))
        self._put(self.tok_pos, np.concatenate(pos))
        self._put(self.tok_slot, np.concatenate(slots))
        self._put(self.gather, np.concatenate(gather))
        self._put(self.req_info, req_info)
        return row, req_info, sample_rows

    # ------------------------------------------------------------------ maps and operand blocks
    def _wmap(self, t, base=None, packed=False):
        if isinstance(t, Mat):
            t = t.data
        if t.dim() == 2:
            rows, k, zdim = t.shape[0], t.shape[1], 1
        else:
            zdim, rows, k = t.shape
        base = base if base is not None else t.data_ptr()
        if t.dtype == torch.uint8:   # e4m3 bytes: byte strides, no swizzle (monoserve/runtime/weights.py:38-40)
            return self.fab.tensor_map(base, [k, rows, zdim], [k, rows * k], [128, 64, 1], dtype=2, swizzle=0, packed=packed)
        return self.fab.tensor_map(base, [k, rows, zdim], [k * 2, rows * k * 2], [64, 64, 1], packed=packed)

    def _amaps(self, t, rows, k):
        """Activation maps of a [rows][k] bf16 buffer for every row-block height."""
        return [self.fab.tensor_map(t.data_ptr(), [k, rows], [k * 2], [64, bm]) for bm in HEIGHTS]

    # ------------------------------------------------------------------ device memory of a build
    def _dev(self, name, **fields):
        """An operand block in the lane's arena."""
        return self.arena.put(pack(name, **fields))

    def _put(self, tensor, values, dtype=np.int32):
        """Write the first len(values) elements of a device tensor without launching a kernel."""
        data = np.ascontiguousarray(values, dtype=dtype)
        if data.size:
            self.fab.write(tensor.data_ptr(), data.tobytes())

    # ------------------------------------------------------------------ stage builders
    def _gemm_split(self, p, wmap, amaps, rows, n_out, k, slabs, parts, label, mark=None, mat=None, bias=None,
                    slab_rows=SPLIT_ROWS):
        """The same product for few rows as `parts` K ranges, every range storing its fp32 partial sums in its own
        slab of `slabs` ([parts][slab_rows][n_out]); the add-norm tile behind it adds the slabs in order.  A 128-row
        weight slice over all of K is a megabyte that one worker streams alone; the ranges spread it over
        parts x n_out / 128 workers, and the sum keeps a defined order (no atomics)."""
        bm = _bm(rows)
        fp8 = mat is not None and mat.fp8
        xm = amaps[HEIGHTS.index(bm)]
        kt = -(-k // 64)
        per = -(-kt // parts)
        ptrs, ranges = [], []
        for q in range(parts):
            k0, kn = q * per, min(per, kt - q * per)
            args = self.arena.put(_C.gemm_args(out=slabs.data_ptr() + 4 * q * slab_rows * n_out, ld_out=n_out, k_tiles=kt,
                                               epi=EPI_F32, bm=bm, n_limit=n_out, w_fp8=int(fp8),
                                               bias=bias.data_ptr() if bias is not None else 0))   # added by the first range
            ptrs.append(args.data_ptr())
            ranges.append(k0 | (kn << 16))
        key = ("split", rows, bm, n_out, parts, kt)
        tmpl = self._templates.get(key)
        if tmpl is None:
            m0, n0 = np.meshgrid(np.arange(0, rows, bm), np.arange(0, n_out, 128), indexing="ij")
            by_range = np.asarray(ranges, dtype=np.int64)[:, None, None]   # (range, row block, slice)
            tmpl = self._templates[key] = tile_array(K_GEMM, i0=n0[None], i1=m0[None], i2=np.minimum(bm, rows - m0)[None],
                                                     a3=by_range)
        per_range = len(tmpl) // parts
        tiles = _retarget(tmpl, a0=np.repeat(np.asarray(ptrs, dtype=np.uint64), per_range), a1=wmap, a2=xm,
                          a4=mat.scale.data_ptr() if fp8 else 0)
        return p.stage(tiles, mark=mark, label=label)

    def _gemm(self, p, wmap, amaps, rows, n_out, k, out, ld_out, epi, label, residual=None, ld_res=0, mark=None,
              mat=None, bias=None, up_offset=0, bm=None, coef=None):
        """A dense GEMM stage: out[rows][n_out] = act[rows][k] x weight[n_out (x2 for SiLU-mul)][k]^T.
        mat: the weight's Mat (e4m3 weights carry their scales into the tiles); bm: the row-block height, when not the
        largest; coef: fp32 per output of the decay epilogue."""
        bm = bm or _bm(rows)
        fp8 = mat is not None and mat.fp8
        args = self.arena.put(_C.gemm_args(
            out=out.data_ptr(), ld_out=ld_out, k_tiles=-(-k // 64), epi=epi, bm=bm, n_limit=n_out,
            residual=residual.data_ptr() if residual is not None else 0, ld_res=ld_res,
            bias=bias.data_ptr() if bias is not None else 0, up_offset=up_offset, w_fp8=int(fp8),
            pair_weight=coef.data_ptr() if coef is not None else 0))
        xm = amaps[HEIGHTS.index(bm)]
        step = 64 if epi in GATED else 128
        key = ("gemm", rows, bm, n_out, step)
        tmpl = self._templates.get(key)
        if tmpl is None:
            m0, n0 = np.meshgrid(np.arange(0, rows, bm), np.arange(0, n_out, step), indexing="ij")
            tmpl = self._templates[key] = tile_array(K_GEMM, i0=n0, i1=m0, i2=np.minimum(bm, rows - m0))
        tiles = _retarget(tmpl, a0=args.data_ptr(), a1=wmap, a2=xm, a4=mat.scale.data_ptr() if fp8 else 0)
        return p.stage(tiles, mark=mark, label=label)

    def _rows(self, kind, args, rows, per):
        key = ("rows", kind, rows, per)
        tmpl = self._templates.get(key)
        if tmpl is None:
            r0 = np.arange(0, rows, per)
            tmpl = self._templates[key] = tile_array(kind, i0=r0, i1=np.minimum(per, rows - r0))
        return _retarget(tmpl, a0=args.data_ptr())

    def _per(self, T):
        """Rows per tile of a stage whose tiles give each exec warp one row at a time: up to four rows per tile
        while that keeps the stage to one round of tiles over the workers (150 tiles on 148 workers are two
        rounds), a multiple of four beyond."""
        nw = self.fab.num_workers
        if T <= 4 * nw:
            return max(1, -(-T // nw))
        return -(-(-(-T // (2 * nw))) // 4) * 4

    def _one(self, kind, args):
        """The single tile of an expand or plan stage."""
        key = ("one", kind)
        tmpl = self._templates.get(key)
        if tmpl is None:
            tmpl = self._templates[key] = tile_array(kind)
        return _retarget(tmpl, a0=args.data_ptr())

    # ------------------------------------------------------------------ request state
    def set_pages(self, slot, pages):
        row = np.zeros(self.bt_stride, dtype=np.int32)
        row[:len(pages)] = pages
        self.fab.write(self.bt.data_ptr() + 4 * slot * self.bt_stride, row.tobytes())

    def set_request(self, slot, seq_len, last_token, temperature=0.0):
        self.fab.write(self.seq_len.data_ptr() + 4 * slot, struct.pack("<i", seq_len))
        self.fab.write(self.last_token.data_ptr() + 4 * slot, struct.pack("<i", last_token))
        self.fab.write(self.steps.data_ptr() + 4 * slot, struct.pack("<i", 0))
        self.fab.write(self.temperature.data_ptr() + 4 * slot, struct.pack("<f", temperature))

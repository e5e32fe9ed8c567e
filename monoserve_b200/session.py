"""A model, its cache and one lane on a resident fabric, stepped by hand: requests bring token ids portion by portion,
and the caller names the places whose logits it wants.  The same lane, programs, page pool and request table as the
serving loop (monoserve_b200/engine.py), without its batching policy or sampling.

    with Session(registry.load(folder), max_tokens=4096) as s:
        logits = s.step("a", [5, 17, 3], want=[0, 2])     # float32 [2, vocab]
        s.end("a")
"""
import time

import numpy as np

from monoserve_b200 import registry
from monoserve_b200.engine import PagePool, RequestTable
from monoserve_b200.fabric import Fabric

SPARE_SMS = 8   # left to the host's copies while the fabric is resident


class Session:
    def __init__(self, model, max_tokens, slots=4, page=16, pass_tokens=2048, max_run_s=3600, keep_residual=False):
        """max_tokens: the most tokens live requests hold at any time; a portion of more than pass_tokens runs as several
        passes."""
        import torch
        n_pages = -(-max_tokens // page) + 2 * slots + 2
        self.page, self.vocab, self.max_positions = page, model.cfg.vocab, getattr(model.cfg, "max_positions", None)
        workers = torch.cuda.get_device_properties(0).multi_processor_count - SPARE_SMS
        self.fab = Fabric(num_workers=workers, pool_bytes=256 << 20)
        self.fab.set_max_run(max_run_s)
        self.kv = model.cache(n_pages, page, slots)
        self.pass_tokens = min(pass_tokens, max(64, max_tokens))
        self.table = RequestTable(self.fab, slots, n_pages)
        extra = {"keep_residual": True} if keep_residual else {}
        self.lane = registry.lane_class(model.cfg)(self.fab, 0, model.cfg, model.weights, self.kv, max_tokens=self.pass_tokens,
                                                   max_slots=slots, bt_stride=n_pages, logit_rows=self.pass_tokens,
                                                   requests=self.table, **extra)
        self.pool, self.free, self.live = PagePool(n_pages), list(range(slots - 1, -1, -1)), {}
        torch.cuda.synchronize()
        self.fab.start()
        self.workers = workers

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()

    def close(self):
        self.fab.stop()
        self.fab.close()

    def _run(self, handle, timeout=120.0):
        before = self.fab.progress()["lanes"][0]["iterations"]
        self.fab.publish(map=[0] * self.workers, caps=[4], order=[0], programs=[handle])
        give_up = time.monotonic() + timeout
        while True:
            p = self.fab.progress()
            if p["error"]:
                raise RuntimeError(f"monofab: device error {p['error']:#x}")
            if p["lanes"][0]["iterations"] > before and not p["lanes"][0]["running"]:
                break
            if time.monotonic() > give_up:
                raise TimeoutError("the fabric did not finish a pass")
            time.sleep(5e-5)
        self.fab.publish(map=[0] * self.workers, caps=[4], order=[0], programs=[0])
        self.fab.release(handle)

    def _reserve(self, r, length):
        need = -(-length // self.page)
        if need > len(r["pages"]):
            r["pages"] += self.pool.take(need - len(r["pages"]))
            self.table.set_pages(r["slot"], r["pages"])

    def step(self, rid, tokens, want=()):
        """Appends `tokens` to request rid (new ids open a request); float32 [len(want), vocab] logits at the wanted
        places among them."""
        if rid not in self.live:
            self.live[rid] = dict(slot=self.free.pop(), pages=[], length=0)
        r = self.live[rid]
        if self.max_positions and r["length"] + len(tokens) > self.max_positions:
            raise ValueError(f"request {rid}: {r['length']} + {len(tokens)} tokens, the model has {self.max_positions} positions")
        self._reserve(r, r["length"] + len(tokens))
        out = []
        for lo in range(0, len(tokens), self.pass_tokens):
            part = tokens[lo:lo + self.pass_tokens]
            places = [w - lo for w in want if lo <= w < lo + len(part)]
            if len(part) == 1 and r["length"] > 0:
                self.lane.set_request(r["slot"], r["length"], part[0])
                self._run(self.lane.build_decode([r["slot"]]))
            else:
                self._run(self.lane.build_prefill([(r["slot"], part, r["length"])], want=[places]))
            r["length"] += len(part)
            if places:
                raw = self.fab.read(self.lane.logits.data_ptr(), 4 * self.vocab * len(places))
                out.append(np.frombuffer(raw, dtype=np.float32).reshape(len(places), self.vocab))
        return np.concatenate(out) if out else np.zeros((0, self.vocab), dtype=np.float32)

    def end(self, rid):
        r = self.live.pop(rid)
        self.pool.give(r["pages"])
        self.free.append(r["slot"])

"""Drives an executor of the stack of mixers step by step, with cache blocks and state slots of its own, and compares the
logits of every new token with a plain forward pass over the sequence's whole history."""
import numpy as np

from logismos_b200.cache import BlockAllocator, SlotAllocator

TOLS = {"float32": 2e-5, "bfloat16": 6e-2}


class Harness:
    """``model``: an executor class with ``parse``; ``pack(cfg, weights)``: its weights; ``forward(cfg, weights, tokens)``:
    the plain logits."""

    def __init__(self, model, pack, forward, cfg, w, dtype, pool_tokens=1024, max_seqs=6, step_tokens=700, block_seed=3, keep_layers=False):
        self.cfg, self.w, self.dtype, self.forward = cfg, w, dtype, forward
        n = pool_tokens // 16
        self.model = model(model.parse(cfg), pack(cfg, w), n, n, step_tokens, max_seqs, max_seqs, dtype=dtype, max_out_rows=step_tokens, keep_layers=keep_layers)
        self.blocks, self.slots, self.hist, self.ref = BlockAllocator(n, n, seed=block_seed), SlotAllocator(max_seqs), {}, {}
        self.seen = self.over = 0
        self.worst = 6.0          # largest error of a bf16 position, in limits

    def expect(self, sid):
        """Reference logits of a sequence's whole history (computed once per history)."""
        h = tuple(self.hist[sid])
        known, z = self.ref.get(sid, ((), None))
        if known[:len(h)] != h:
            z = self.forward(self.cfg, self.w, h)
            self.ref[sid] = (h, z)
        return z[:len(h)]

    def run(self, entries, check=True):
        """entries: (sequence, tokens); every new token's logits are compared."""
        ids, cached, new, tabs, sl = [], [], [], [], []
        for sid, toks in entries:
            prev = self.hist.setdefault(sid, [])
            cached.append(len(prev)); new.append(len(toks)); ids.extend(int(t) for t in toks)
            prev.extend(int(t) for t in toks)
            tabs.append(self.blocks.ensure(sid, len(prev))); sl.append(self.slots.get(sid))
        toks = self.model.step(ids, cached, new, np.stack(tabs), sl, out_rows=range(len(ids)))
        assert self.model.device_status() == 0
        z, at = self.model.last_logits(), 0
        assert np.array_equal(toks, z.argmax(1))
        for (sid, t) in entries:
            if check:
                ref = self.expect(sid)
                self.compare(z[at:at + len(t)], ref[len(ref) - len(t):], (sid, len(ref)), ref)
            at += len(t)
        return z

    def compare(self, z, ref, what, scale=None, factor=1.0):
        """fp32: every position. bf16: a position whose output is nearly zero before a norm, or whose router nearly ties, can
        be moved far by rounding alone, so single ones may exceed the limit (``close`` counts them over the whole test)."""
        err = np.sqrt(np.mean((z - ref) ** 2, axis=1)) / np.sqrt(np.mean((ref if scale is None else scale) ** 2))
        bound = factor * TOLS[self.dtype]
        self.seen += err.size
        self.over += int((err > bound).sum())
        assert err.max() <= (bound if self.dtype == "float32" else self.worst * bound), (what, int(err.argmax()), float(err.max()))

    def close(self):
        self.model.close()
        assert self.over <= 0.02 * self.seen, (self.over, self.seen)

    def known(self, sid, tokens):
        """Computes the reference of a sequence's full history once, before it is fed in parts."""
        self.hist[sid] = [int(t) for t in tokens]
        self.expect(sid)
        self.hist[sid] = []

    def drop(self, sid):
        self.blocks.release(sid); self.slots.release(sid); self.hist.pop(sid)


def tokens(rng, cfg, n):
    return rng.integers(0, cfg["vocab"], n)


def greedy_reference(forward, cfg, w, prompt, n):
    """The greedy continuation and its smallest margin."""
    h = list(prompt)
    margins = []
    for _ in range(n):
        z = forward(cfg, w, h)[-1]
        top = np.sort(z)[-2:]
        margins.append(top[1] - top[0])
        h.append(int(z.argmax()))
    return h[len(prompt):], min(margins)

"""Several sequences on one model: token portions in, logits out.

`Sequences` owns what the sequences keep on the device.  A sequence takes a set of caches (one per layer run) when its
first tokens arrive and gives it back when it ends; the next sequence gets the set emptied, together with the captured
one-token step that belongs to its pointers.  A portion of several tokens runs as a prompt pass, a single token as a
replay of the captured step.
"""
import torch

from . import archs
from . import dev_residency as dr
from . import prefill as pf


class _Slot:
    def __init__(self, w, cfg):
        self.kv = [None] * archs.of(cfg).n_slots(cfg)
        self.runner = dr.GraphRunner(w, cfg, self.kv)
        self.length = 0


class Sequences:
    def __init__(self, w, cfg, max_tokens=None):
        self.w, self.cfg = w, cfg
        self.arch = archs.of(cfg)
        if max_tokens is not None:
            dr._KV_MAX_SEQ = max(dr._KV_MAX_SEQ, int(max_tokens))
        self.live = {}
        self.free = []

    def _slot(self, sid):
        s = self.live.get(sid)
        if s is None:
            s = self.free.pop() if self.free else _Slot(self.w, self.cfg)
            self.live[sid] = s
        return s

    def length(self, sid):
        return self.live[sid].length if sid in self.live else 0

    def step(self, sid, tokens, want=()):
        """Run the next tokens of sequence `sid`; logits [len(want), vocab] of the wanted places among them (None when
        nothing is wanted)."""
        n = len(tokens)
        if n == 0:
            if len(want):
                raise ValueError("logits wanted of an empty portion")
            return None
        if any(not 0 <= int(p) < n for p in want):
            raise ValueError(f"wanted places {list(want)} of {n} tokens")
        V = self.cfg.get("vocab")
        if V is not None and any(not 0 <= int(t) < V for t in tokens):
            raise ValueError("token id outside the vocabulary")
        s = self._slot(sid)
        for c in s.kv:
            if isinstance(c, dr.DeviceGroupedKV):
                c.require(n)
        out = {}
        if n == 1:
            lg = self._one(s, int(tokens[0]))
            out[0] = lg.reshape(-1)
        else:
            toks = torch.tensor([int(t) for t in tokens], dtype=torch.long)
            for c0 in range(0, n, self.arch.max_rows):
                part = toks[c0:c0 + self.arch.max_rows]
                rows = sorted({int(p) - c0 for p in want if c0 <= int(p) < c0 + part.numel()})
                lg = pf.prefill_resident(self.w, self.cfg, part, s.kv, want_rows=rows)
                out.update({c0 + r: lg[i] for i, r in enumerate(rows)})
        s.length += n
        if not len(want):
            return None
        return torch.stack([out[int(p)] for p in want])

    def _one(self, s, tok):
        if not s.runner.captured:
            if any(c is None for c in s.kv) or not getattr(s, "seeded", False):
                s.seeded = True
                return s.runner.seed(torch.tensor([tok]), torch.tensor([s.length]))    # eager; settles every pointer
            s.runner.capture(torch.tensor([tok]), torch.tensor([s.length]))
        return s.runner.replay_logits(tok)

    def end(self, sid):
        """The sequence is finished; what it held is free again."""
        s = self.live.pop(sid, None)
        if s is None:
            return
        s.runner.stream.synchronize()
        for c in s.kv:
            if c is not None:
                c.reset()
        torch.cuda.synchronize()
        s.length = 0
        self.free.append(s)

"""Sequences on one stage that holds a whole model: slots, micro-batches, greedy generation.

A stage keeps n_seq cache / state slots.  The engine gives a request a slot when its first tokens come and takes it
back when the request ends, cuts what it is fed into micro-batches of the stage's n_ubatch tokens, and in a decode
round runs requests that stand at the same position in neighbouring slots as one batch.  Works on every stage, the
K-quant decoder's and those whose layers are described one by one.
"""
from __future__ import annotations

import os

import numpy as np
import torch

from .capi import PRECISION_BF16, PRECISION_F32
from .stage import Stage

PRECISIONS = {"bfloat16": PRECISION_BF16, "float32": PRECISION_F32}


class PrecisionError(ValueError):
    """the model does not run in the precision asked for"""


def open_stage(path, precision="bfloat16", **kw):
    """Stage with the whole model at `path`: a checkpoint folder, or a GGUF file (K-quant weights, which have no
    32-bit mode).  kw: n_ctx, n_seq, n_ubatch, device."""
    if os.path.isdir(path):
        from .checkpoint import Checkpoint

        with Checkpoint(path) as ck:
            return Stage.from_checkpoint(ck, precision=PRECISIONS[precision], **kw)[0]
    if precision != "bfloat16":
        raise PrecisionError("a GGUF model runs on its quantised weights; it has no 32-bit mode")
    from .gguf import GgufFile

    with GgufFile(path) as g:
        return Stage.from_gguf(g, **kw)[0]


class Request:
    def __init__(self, slot):
        self.slot, self.pos = slot, 0


class Engine:
    def __init__(self, stage):
        c = stage.cfg
        if not (c.has_embd and c.has_output):
            raise ValueError("the engine needs a stage with the embedding and the output head")
        self.stage, self.n_ctx, self.n_ubatch, self.n_vocab = stage, c.n_ctx, c.n_ubatch, c.n_vocab
        self.free = list(range(c.n_seq))
        self.live = {}
        self.n_seq = c.n_seq
        dev = stage.device
        # fixed buffers: a decode step's captured graph is looked up by its pointers
        self._tok = torch.zeros(c.n_seq, dtype=torch.int32, device=dev)
        self._next = torch.zeros(c.n_seq, dtype=torch.int32, device=dev)
        self._logits = torch.empty((c.n_seq, c.n_vocab), dtype=torch.float32, device=dev)

    # ---- requests -------------------------------------------------------------------------------
    def start(self, rid):
        if rid in self.live:
            raise ValueError(f"request {rid!r} is live already")
        if not self.free:
            raise RuntimeError("no free sequence slot")
        self.live[rid] = Request(self.free.pop(0))
        return self.live[rid]

    def end(self, rid):
        """the request's slot goes back; the next sequence in it starts at position 0 and reads nothing of this one"""
        self.free.append(self.live.pop(rid).slot)
        self.free.sort()

    def feed(self, rid, tokens, want=()):
        """Runs a request's next tokens; -> logits [len(want), n_vocab] (host, f32) at the places `want` among them.
        The request is started if it is new."""
        tokens = np.asarray(tokens, dtype=np.int64).reshape(-1)
        want = [int(i) for i in want]
        n = len(tokens)
        if n and (tokens.min() < 0 or tokens.max() >= self.n_vocab):
            raise ValueError("token id outside the vocabulary")
        if any(i < 0 or i >= n for i in want):
            raise ValueError("wanted place outside the tokens")
        r = self.live.get(rid) or self.start(rid)
        if r.pos + n > self.n_ctx:
            raise ValueError(f"request {rid!r} would hold {r.pos + n} tokens, the cache has room for {self.n_ctx}")
        out = np.empty((len(want), self.n_vocab), np.float32)
        for lo in range(0, n, self.n_ubatch):
            hi = min(n, lo + self.n_ubatch)
            rows = [(k, i - lo) for k, i in enumerate(want) if lo <= i < hi]
            last_only = all(i == hi - lo - 1 for _, i in rows)
            lg = self._forward(r, tokens[lo:hi], not last_only)
            if rows:
                host = lg.cpu().numpy()
                for k, i in rows:
                    out[k] = host[0 if last_only else i]
        return out

    def _forward(self, r, tokens, all_logits):
        T = len(tokens)
        if T == 1:
            tok, lg = self._tok[:1], self._logits[:1]
            tok.copy_(torch.from_numpy(tokens.astype(np.int32)))
        else:
            tok = torch.from_numpy(tokens.astype(np.int32)).to(self.stage.device)
            lg = torch.empty((T, self.n_vocab), dtype=torch.float32, device=self.stage.device) if all_logits else self._logits[:1]
        nxt = self._next[:1] if not all_logits or T == 1 else torch.empty(T, dtype=torch.int32, device=self.stage.device)
        self.stage.forward(tokens=tok, n_seq=1, T=T, pos0=r.pos, logits=lg, all_logits=all_logits and T > 1, next_tokens=nxt,
                           seq0=r.slot)
        r.pos += T
        return lg

    def check(self):
        """raises if a bounded device-side wait gave up since the last call"""
        self.stage.synchronize()

    # ---- greedy generation ----------------------------------------------------------------------
    def decode_groups(self, rids):
        """live requests as runs of neighbouring slots at one position: each run is one batch"""
        groups = []
        for rid in sorted(rids, key=lambda i: self.live[i].slot):
            r = self.live[rid]
            if groups:
                p = self.live[groups[-1][-1]]
                if p.slot + 1 == r.slot and p.pos == r.pos and len(groups[-1]) < self.n_ubatch:
                    groups[-1].append(rid)
                    continue
            groups.append([rid])
        return groups

    def generate(self, prompts, max_new, stop=()):
        """Greedy continuation of every prompt (lists of token ids): -> list of lists of new ids, at most max_new each,
        ending early after an id in `stop`.  More prompts than slots wait for one to become free."""
        stop = set(int(t) for t in stop)
        out = [[] for _ in prompts]
        waiting = list(range(len(prompts)))
        running = {}
        last = np.zeros(len(prompts), np.int32)

        def emit(i, token):
            out[i].append(int(token))
            last[i] = token
            if len(out[i]) >= max_new or int(token) in stop:
                self.end(("gen", i))
                running.pop(i)

        while waiting or running:
            while waiting and self.free and max_new > 0:
                i = waiting.pop(0)
                if not len(prompts[i]):
                    raise ValueError("a prompt needs at least one token")
                running[i] = ("gen", i)
                lg_last = self.feed(("gen", i), prompts[i])  # noqa: F841 - the last position's greedy id is on the device
                emit(i, int(self._next[0].item()))
            if max_new <= 0:
                break
            if waiting and not running:
                raise RuntimeError("no free sequence slot")
            for group in self.decode_groups(list(running.values())):
                ids = [rid[1] for rid in group]
                r0, n = self.live[group[0]], len(group)
                if r0.pos + 1 > self.n_ctx:
                    raise ValueError(f"a sequence would hold more than {self.n_ctx} tokens")
                tok = self._tok[:n]
                tok.copy_(torch.from_numpy(last[ids]))
                self.stage.forward(tokens=tok, n_seq=n, T=1, pos0=r0.pos, logits=self._logits[:n], next_tokens=self._next[:n],
                                   seq0=r0.slot)
                for rid in group:
                    self.live[rid].pos += 1
                nxt = self._next[:n].cpu().numpy()
                for i, t in zip(ids, nxt):
                    emit(i, t)
        self.check()
        return out

"""Sequences on a model's slots: opening and closing them, feeding tokens in portions, and generation.

`Session` hands a model's cache / state slots to named sequences and runs portions of any length through the model's own
passes.  `generate` serves prompts: each prompt in portions, then one step per token for all sequences together (models
whose steps know every slot's position, replayed from one CUDA graph when the choice is greedy) or sequence by sequence.
"""
from __future__ import annotations

import numpy as np

from . import ops
from .layered import POS_NEXT, LayeredDecoder


class Session:
    def __init__(self, model):
        self.model, self.torch = model, model.torch
        self._free = list(range(model.max_batch))[::-1]
        self._slots, self._lengths = {}, {}

    def __contains__(self, name) -> bool:
        return name in self._slots

    def open(self, name) -> int:
        if name in self._slots:
            raise ops.ArgumentException(f"sequence '{name}' is open")
        if not self._free:
            raise ops.InvalidOperationException(f"all {self.model.max_batch} sequence slots are in use")
        slot = self._free.pop()
        self.model.reset_sequence(slot)
        self._slots[name], self._lengths[name] = slot, 0
        return slot

    def close(self, name):
        slot = self._slots.pop(name)
        del self._lengths[name]
        self.model.reset_sequence(slot)
        self._free.append(slot)

    def length(self, name) -> int:
        return self._lengths[name]

    def slot(self, name) -> int:
        return self._slots[name]

    def feed(self, name, tokens, want=()):
        """Appends `tokens` to the sequence; returns the logits [len(want), vocab] (CUDA) at the places `want` among them,
        or None when nothing is wanted."""
        t, m = self.torch, self.model
        tokens = np.ascontiguousarray(tokens, np.int32)
        want = np.asarray(want, np.int64)
        if tokens.size == 0:
            raise ops.ArgumentException("feed: no tokens")
        if want.size and (want.min() < 0 or want.max() >= tokens.size):
            raise ops.ArgumentOutOfRangeException(f"feed: a wanted place outside the {tokens.size} tokens")
        if tokens.min() < 0 or tokens.max() >= m.cfg["vocab"]:
            raise ops.ArgumentOutOfRangeException(f"feed: a token outside the vocabulary of {m.cfg['vocab']}")
        out = t.empty((want.size, m.cfg["vocab"]), dtype=t.float32, device="cuda") if want.size else None
        dev = t.from_numpy(tokens).cuda()
        pos = self._lengths[name]
        for lo in range(0, tokens.size, m.max_chunk):
            hi = min(lo + m.max_chunk, tokens.size)
            here = np.nonzero((want >= lo) & (want < hi))[0]
            rows = t.from_numpy((want[here] - lo).astype(np.int32)).cuda() if here.size else None
            logits = m.forward_rows(dev[lo:hi], pos + lo, self._slots[name], rows)
            if logits is not None:
                out[t.from_numpy(here).cuda()] = logits
            self._lengths[name] = pos + hi
        return out


class Sampling:
    """How the next token is picked: temperature 0 is the greedy choice; the other fields are the device sampler's."""

    def __init__(self, temperature: float = 0.0, top_k: int = 0, top_p: float = 1.0, min_p: float = 0.0, repetition_penalty: float = 1.0,
                 window: int = 64, seed: int = 0):
        self.temperature, self.top_k, self.top_p, self.min_p = temperature, top_k, top_p, min_p
        self.repetition_penalty, self.window, self.seed = repetition_penalty, window, seed

    @property
    def greedy(self) -> bool:
        return self.temperature <= 0 and self.repetition_penalty == 1.0


def generate(model, prompts, max_new: int, sampling: Sampling | None = None, graph: bool = True):
    """`max_new` tokens after each of `prompts` (lists of token ids, up to the model's slot count); a list of lists."""
    t, sampling = model.torch, sampling or Sampling()
    B = len(prompts)
    if not 0 < B <= model.max_batch:
        raise ops.ArgumentException(f"{B} prompts for {model.max_batch} sequence slots")
    if max_new <= 0:
        return [[] for _ in prompts]
    if max(len(p) for p in prompts) + max_new > model.cfg["max_seq"]:
        raise ops.ArgumentOutOfRangeException(f"prompt and {max_new} new tokens exceed {model.cfg['max_seq']} positions")
    dev, rng = ops.DeviceOps(model.ctx), np.random.default_rng(sampling.seed)
    session, history = Session(model), [list(p) for p in prompts]
    for i, p in enumerate(prompts):
        if session.open(i) != i:
            raise ops.InvalidOperationException("generate needs the model's slots in order")
    logits = t.cat([session.feed(i, p, [len(p) - 1]) for i, p in enumerate(prompts)])

    def pick(rows):
        if sampling.repetition_penalty != 1.0:
            w = max(1, sampling.window)
            ids = np.full((B, w), -1, np.int32)
            for i, hist in enumerate(history):
                tail = hist[-w:]
                ids[i, :len(tail)] = tail
            dev.repetition_penalty_(rows, t.from_numpy(ids).cuda(), sampling.repetition_penalty)
        if sampling.temperature <= 0:
            return dev.argmax(rows)
        u = t.from_numpy(rng.random(B, dtype=np.float32)).cuda()
        return dev.sample(rows, sampling.temperature, sampling.top_k, sampling.top_p, sampling.min_p, uniform=u)

    def note(toks):
        for i, v in enumerate(toks.cpu().tolist()):
            history[i].append(v)

    tok = pick(logits)
    note(tok)
    if isinstance(model, LayeredDecoder):
        nxt = t.empty_like(tok)
        if sampling.greedy and graph and max_new > 2:
            # the step reads its tokens from where the last one left them and advances the positions on the device
            model.step(tok, POS_NEXT, logits=logits, argmax=nxt)
            tok.copy_(nxt)
            note(tok)
            out = t.empty((max_new - 2, B), dtype=t.int32, device="cuda")
            g = t.cuda.CUDAGraph()
            with t.cuda.graph(g):
                model.step(tok, POS_NEXT, logits=logits, argmax=nxt)
                tok.copy_(nxt)
            for k in range(max_new - 2):
                g.replay()
                out[k].copy_(nxt)
            for row in out:
                note(row)
        else:
            for _ in range(max_new - 1):
                model.step(tok, POS_NEXT, logits=logits, argmax=nxt)
                tok = nxt.clone() if sampling.greedy else pick(logits)
                note(tok)
    else:
        for _ in range(max_new - 1):
            rows = t.cat([session.feed(i, [hist[-1]], [0]) for i, hist in enumerate(history)])
            tok = pick(rows)
            note(tok)
    for i in range(B):
        session.close(i)
    return [hist[len(p):] for hist, p in zip(history, prompts)]

"""Checks that any design's tests can run against its plain implementation: a model folder, the plain module's two functions and an
engine on the stand-in kernels (CPU) or the CUDA kernels (GPU)."""
import os
import random

import torch

from mini_inference_b200.engine.batch import StepEntry
from mini_inference_b200.engine.factory import load_model, make_runner
from mini_inference_b200.weights.safetensors_io import write_safetensors
from tests.ref_ops import TorchRefOps


class Judge:
    """The plain implementation's logits of a model folder (its weights are read once)."""

    def __init__(self, plain):
        self.plain, self._weights = plain, {}

    def forget(self, d):
        self._weights.pop(d, None)

    def logits(self, d, ids):
        if d not in self._weights:
            self._weights[d] = self.plain.load_model_dir(d)
        cfg, w = self._weights[d]
        return self.plain.forward_logits(cfg, w, ids).float()

    def greedy(self, d, prompt, n):
        ids = list(prompt)
        for _ in range(n):
            ids.append(int(self.logits(d, ids)[-1].argmax()))
        return ids[len(prompt):]


def rewrite_weights(d, plain, change):
    """Replaces the tensors for which change(name, tensor) gives values."""
    _, w = plain.load_model_dir(d, dtype=torch.bfloat16)
    for name in w:
        new = change(name, w[name])
        if new is not None:
            w[name] = new.to(torch.bfloat16)
    write_safetensors(os.path.join(d, "model.safetensors"), [(n, tuple(t.shape), t.dtype, (lambda t=t: t)) for n, t in w.items()])
    return d


def tokens(vocab, n, seed):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(n)]


def err(got, want):
    return ((got - want).abs().max() / want.abs().max()).item()


def assert_close(got, want, tol, what=""):
    """float32 (tol < 1e-2): every logit within tol of the largest.  bfloat16: the root mean square over the vocabulary within tol at
    every position and within a third of it at the median one."""
    if tol < 1e-2:
        assert err(got, want) < tol, (what, err(got, want))
        return
    per = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    assert per.max().item() < tol and per.median().item() < tol / 3, (what, per.median().item(), per.max().item())


def engine(d, page, pages, dtype="float32", device="cpu", max_seqs=4):
    _, model, _ = load_model(d, dtype, device)
    return make_runner(model, page, pages, max_seqs, ops=TorchRefOps() if device == "cpu" else None)


def feed(runner, key, ids, cuts):
    """ids in portions of the given sizes, all logits wanted: [n, vocab]."""
    seq = runner.cache.admit(key)
    out, at = [], 0
    for n in cuts:
        out.append(runner.step([StepEntry(seq, ids[at:at + n], range(n))]).float().cpu())
        at += n
        runner.cache.check_invariants()
    assert at == len(ids)
    runner.cache.free(seq)
    return torch.cat(out)


def portions(n, rng, smallest=2, largest=9):
    cuts = []
    while n > 0:
        c = min(n, rng.randint(smallest, largest))
        if n - c == 1:
            c += 1
        cuts.append(c)
        n -= c
    return cuts


def check_cuts(runner, judge, d, vocab, tol, n=75):
    """Whole prompt; most of it then the last 24 one by one; portions of 2..9 tokens; portions of two; from the first token one by
    one (long decoding: every cache row and every state is written one token at a time)."""
    ids = tokens(vocab, n, seed=3)
    want = judge.logits(d, ids)
    free = runner.cache.free_pages()
    assert_close(feed(runner, "w", ids, [n]), want, tol, "whole")
    assert_close(feed(runner, "d", ids, [n - 24] + [1] * 24), want, tol, "decode")
    assert_close(feed(runner, "p", ids, portions(n, random.Random(1))), want, tol, "portions")
    assert_close(feed(runner, "2", ids[:20], [2] * 10), want[:20], tol, "twos")
    assert_close(feed(runner, "1", ids, [1] * n), want, tol, "ones")
    runner.cache.check_invariants()
    assert runner.cache.free_pages() == free


def check_mixed(make, judge, d, vocab, page, tol, lens=(23, 9, 31, 17, 40, 12, 27, 36, 20, 33), seed=7):
    """Up to four live requests, portions of some beside single tokens of others, some left out of a step; the pool holds four of
    the longest requests and there are four slots, so pages and slots are used again (both counted)."""
    rng = random.Random(seed)
    reqs = {f"r{i}": tokens(vocab, n, seed=100 + i) for i, n in enumerate(lens)}
    want = {k: judge.logits(d, v) for k, v in reqs.items()}
    pages = 4 * -(-max(lens) // page)
    runner = make(pages)
    takes, slot_uses = {}, {}
    for g in runner.cache.kv_groups:
        inner = g.pool.take
        def counted(inner=inner, gi=id(g)):
            pg = inner()
            takes[(gi, pg)] = takes.get((gi, pg), 0) + 1
            return pg
        g.pool.take = counted
    pending, live, got = list(reqs), {}, {k: [] for k in reqs}
    while pending or live:
        while pending and len(live) < 4:
            k = pending.pop(0)
            live[k] = [runner.cache.admit(k), 0]
            slot_uses[live[k][0].slot] = slot_uses.get(live[k][0].slot, 0) + 1
        entries, owners = [], []
        for k, (seq, at) in live.items():
            if rng.random() < 0.2 and len(live) > 1:
                continue
            left = len(reqs[k]) - at
            n = 1 if (at > 0 and rng.random() < 0.5) else min(left, rng.randint(2, 8))
            if left - n == 1:
                n = left
            entries.append(StepEntry(seq, reqs[k][at:at + n], range(n)))
            owners.append((k, n))
        if not entries:
            continue
        logits = runner.step(entries).float().cpu()
        row = 0
        for k, n in owners:
            got[k].append(logits[row:row + n])
            row += n
            live[k][1] += n
        for k in [k for k, (seq, at) in live.items() if at == len(reqs[k])]:
            runner.cache.free(live.pop(k)[0])
        runner.cache.check_invariants()
    for k in reqs:
        assert_close(torch.cat(got[k]), want[k], tol, k)
    assert runner.cache.free_pages() == pages
    assert len(slot_uses) <= 4 and max(slot_uses.values()) >= 2, "no slot was used again"
    if takes:
        assert sum(n - 1 for n in takes.values()) * 3 >= sum(takes.values()), "too few pages were used again"

"""Fetodra in the engine against the plain implementation (tests/plain/fetodra_plain.py).

Without a GPU the engine runs on the stand-in kernel namespace (tests/ref_ops.py), which exercises configuration,
weights, spec, parts, the cache manager, the batch builder, the scheduler and the entry point.  With a GPU
(-m gpu) the same checks run on the CUDA kernels in float32 and bfloat16, plus each kernel alone against the plain
statement of its op."""
import io
import json
import math
import os
import random
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from mini_inference_b200 import LLM, SamplingParams
from mini_inference_b200.cache.manager import CacheManager
from mini_inference_b200.config import ConfigError, load_config, resolve
from mini_inference_b200.config.fetodra_config import FetodraConfig
from mini_inference_b200.engine.batch import StepEntry
from mini_inference_b200.engine.factory import load_model, make_runner
from mini_inference_b200.parts.base import KVCacheNeed
from mini_inference_b200.weights import write_random_model
from mini_inference_b200.weights.safetensors_io import write_safetensors
from tests.plain import fetodra_plain as plain
from tests.ref_ops import TorchRefOps

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
gpu = pytest.mark.gpu


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def attn(heads, kv, dim, vdim, window, keep, mlp=None, conv=3, rot=4, base=500.0, scale=0.3, cap=6.0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "softcap": cap,
         "rot": {"base": base, "dims": rot}, "mask": {"size": window, "keep_first": keep}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mamba(heads, vdim, state, groups, parts, conv=4, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": parts, "conv": conv}}


def config(width, vocab, layers, eps=1e-5, alpha=1.5):
    return {"architecture": "Fetodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


# Small configurations that differ from one another in every size; none makes two sizes equal by accident.
CONFIGS = {
    # borrowed keys with a wider window, more kept keys, another cap, scale and number of taps than the layer that owns them (and one with
    # a narrower window); value rows of another size than key rows; Mamba-2 with groups and norm parts, with a feed-forward and without
    "mix": (config(48, 131, [attn(6, 2, 8, 12, 9, 2, dense(40, 0.8)), mamba(4, 6, 10, 2, 3), attn(4, 4, 12, 8, 7, 5, conv=2, rot=12, base=90.0),
                             attn(6, 2, 8, 12, 15, 6, dense(28, 2.5), conv=4, scale=0.5, cap=3.0, kv_from=0),
                             mamba(6, 4, 7, 3, 1, conv=2, mlp=dense(36, 1.3)), attn(6, 2, 8, 12, 5, 1, conv=2, cap=9.0, kv_from=0)]), 4),
    # one head, one group, one tap, nothing kept, a window of one key, no feed-forward anywhere, alpha of 1, a state of one number a channel
    "ones": (config(40, 97, [attn(1, 1, 24, 24, 1, 0, conv=1, rot=2), mamba(1, 20, 1, 1, 1, conv=1), attn(1, 1, 16, 16, 6, 1, conv=1, rot=16),
                             mamba(3, 8, 5, 3, 3, conv=2)], eps=1e-6, alpha=1.0), 8),
    # pages of 16, heads of 64 and 128 and states of 64 and 128 rows (the sizes the tensor-core kernels take); windows that end inside a
    # tile; kept keys that end inside and at the edge of a page, more than a page of them for the borrower
    "pages": (config(64, 150, [attn(4, 2, 64, 64, 37, 5, dense(72, 1.1), conv=4, rot=32, base=1e4, scale=0.125, cap=10.0), mamba(2, 32, 64, 1, 2, mlp=dense(24, 3.0)),
                               attn(4, 2, 64, 64, 50, 21, conv=3, rot=32, base=1e4, scale=0.2, cap=4.0, kv_from=0),
                               attn(3, 1, 128, 128, 30, 16, dense(36, 0.6), conv=2, rot=64, base=3e5, scale=0.09, cap=25.0), mamba(2, 64, 128, 2, 1, conv=3)], alpha=2.5), 16),
}
STD = 0.25


def _perturb(d, seed=7):
    """The random-weights writer leaves biases, decays and the norms' offsets at zero and the short filters small; give every one of them
    values, so that leaving one out shows, and states that remember hundreds of tokens (small steps)."""
    cfg, w = plain.load_model_dir(d, dtype=torch.bfloat16)
    g = torch.Generator().manual_seed(seed)
    rnd = lambda t, s: torch.randn(t.shape, generator=g) * s      # noqa: E731
    for name in w:
        if name.endswith((".b", ".norm1", ".norm2", "final.norm")):
            w[name] = rnd(w[name], 0.3).to(torch.bfloat16)
        elif name.endswith(".conv"):
            w[name] = (rnd(w[name], 0.5) + 0.2).to(torch.bfloat16)
        elif name.endswith("dt_bias"):
            w[name] = (rnd(w[name], 1.0) - 2.5).to(torch.bfloat16)
        elif name.endswith("A_log"):
            w[name] = (rnd(w[name], 0.7) - 1.0).to(torch.bfloat16)
    write_safetensors(os.path.join(d, "model.safetensors"), [(n, tuple(t.shape), t.dtype, (lambda t=t: t)) for n, t in w.items()])
    _PLAIN.pop(d, None)
    return d


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    out = {}
    for i, (name, (cfg, page)) in enumerate(CONFIGS.items()):
        d = str(tmp_path_factory.mktemp("fetodra_" + name))
        write_random_model(cfg, d, seed=70 + i, std=STD, norm_init="uniform")
        out[name] = (_perturb(d), cfg, page)
    return out


def tokens(vocab, n, seed):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(n)]


_PLAIN = {}


def plain_logits(d, ids):
    if d not in _PLAIN:
        _PLAIN[d] = plain.load_model_dir(d)
    cfg, w = _PLAIN[d]
    return plain.forward_logits(cfg, w, ids).float()


def err(got, want):
    return ((got - want).abs().max() / want.abs().max()).item()


def assert_close(got, want, tol, what=""):
    """float32 (tol < 1e-2): every logit within tol of the largest.  bfloat16: the root mean square over the vocabulary within tol at
    every position and within a fifth of it at the median one (the norms behind the sums pass a rounding on undamped, and the stand-in
    kernels in bfloat16 show the same largest error at the same position)."""
    if tol < 1e-2:
        assert err(got, want) < tol, (what, err(got, want))
        return
    per = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    assert per.max().item() < tol and per.median().item() < tol / 5, (what, per.median().item(), per.max().item())


def engine(d, page, pages, dtype="float32", device="cpu", max_seqs=4):
    _, model, _ = load_model(d, dtype, device)
    return make_runner(model, page, pages, max_seqs, ops=TorchRefOps() if device == "cpu" else None)


def feed(runner, key, ids, cuts):
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


def check_cuts(runner, d, vocab, tol, n=75):
    """Whole prompt; most of it then the last 24 one by one; portions of 2..9 tokens; portions of two; from the first token one by
    one (long decoding: every cache row, every state is written one token at a time, every window passes over decoded tokens)."""
    ids = tokens(vocab, n, seed=3)
    want = plain_logits(d, ids)
    free = runner.cache.free_pages()
    assert_close(feed(runner, "w", ids, [n]), want, tol, "whole")
    assert_close(feed(runner, "d", ids, [n - 24] + [1] * 24), want, tol, "decode")
    assert_close(feed(runner, "p", ids, portions(n, random.Random(1))), want, tol, "portions")
    assert_close(feed(runner, "2", ids[:20], [2] * 10), want[:20], tol, "twos")
    assert_close(feed(runner, "1", ids, [1] * n), want, tol, "ones")
    runner.cache.check_invariants()
    assert runner.cache.free_pages() == free


def check_mixed(make, d, vocab, page, tol, lens=(23, 9, 31, 17, 40, 12, 27, 36, 20, 33), seed=7):
    """Up to four live requests, portions of some beside single tokens of others, some left out of a step; the pool holds four of
    the longest requests and there are four slots, so pages and slots are used again (both counted)."""
    rng = random.Random(seed)
    reqs = {f"r{i}": tokens(vocab, n, seed=100 + i) for i, n in enumerate(lens)}
    want = {k: plain_logits(d, v) for k, v in reqs.items()}
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
    assert sum(n - 1 for n in takes.values()) * 3 >= sum(takes.values()), "too few pages were used again"


# ---------------------------------------------------------------- configuration, registry, spec, cache needs
def test_config_reads_every_key_and_refuses_what_is_missing():
    raw = CONFIGS["mix"][0]
    assert resolve(raw).name == "Fetodra" and resolve({"architectures": ["Fetodra"]}).name == "Fetodra"
    cfg = FetodraConfig.from_dict(raw)
    assert FetodraConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.postln_alpha == 1.5 and cfg.layers[0].mlp.limit == 0.8 and cfg.layers[1].mlp is None and cfg.layers[4].mlp.ff == 36
    assert cfg.layers[3].mixer_dict()["kv_from"] == 0 and "kv_from" not in cfg.layers[0].mixer_dict()
    assert cfg.layers[3].mixer_dict()["mask"] == {"size": 15, "keep_first": 6}
    for path, msg in ((("norm",), "norm"), (("postln_alpha",), "postln_alpha"), (("layers", 0, "mixer", "conv"), "conv"), (("layers", 0, "mixer", "vdim"), "vdim"),
                      (("layers", 0, "mixer", "rot", "base"), "base"), (("layers", 0, "mixer", "mask", "size"), "size"), (("layers", 0, "mixer", "scale"), "scale"),
                      (("layers", 1, "mixer", "norm_groups"), "norm_groups"), (("layers", 1, "mixer", "state"), "state"), (("layers", 0, "mlp", "limit"), "limit")):
        broken = json.loads(json.dumps(raw))
        node = broken
        for p in path[:-1]:
            node = node[p]
        del node[path[-1]]
        with pytest.raises(ConfigError, match=msg):
            FetodraConfig.from_dict(broken)
    for edit, msg in ((lambda c: c["layers"][0].update(type="retention"), "retention"), (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
                      (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"), (lambda c: c["layers"][5]["mixer"].update(kv_from=3), "kv_from"),
                      (lambda c: c["layers"][3]["mixer"].update(vdim=8), "vdim"), (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
                      (lambda c: c["layers"][3]["mixer"]["rot"].update(base=1.0), "rot"), (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "dims"),
                      (lambda c: c["layers"][1]["mixer"].update(groups=3), "groups"), (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
                      (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "softcap"), (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe")):
        bad = json.loads(json.dumps(raw))
        edit(bad)
        with pytest.raises(ConfigError, match=msg):
            FetodraConfig.from_dict(bad)


def test_spec_order_and_cache_needs(dirs):
    d, cfg, page = dirs["mix"]
    _, spec = load_config(d)
    assert spec.residual == "float32" and [s.cache_from for s in spec.order] == [None, None, None, 0, None, 0]
    assert [layer.block for layer in spec.layers] == ["postnorm", "postnorm_mixer", "postnorm_mixer", "postnorm", "postnorm", "postnorm_mixer"]
    assert spec.layers[0].part("norm1").get("alpha") == 1.5 and spec.layers[3].part("mixer").get("borrows_keys")
    runner = engine(d, page, 8)
    needs = [g.need for g in runner.cache.kv_groups]
    # the pages that layers 0, 3 and 5 read are kept for the widest window and the longest kept start among them
    assert needs == [KVCacheNeed(2, 8, 15, value_dim=12, keep_first=6), KVCacheNeed(4, 12, 7, value_dim=8, keep_first=5)]
    caches = runner.cache.layer_caches
    assert caches[0].k.shape[-1] == 8 and caches[0].v.shape[-1] == 12
    assert caches[3].k is None and caches[3].group == -1                       # no pages of its own ...
    assert caches[3].state.shape == (5, 3 * 48) and caches[0].state.shape == (5, 2 * (48 + 16 + 24)) and caches[5].state.shape == (5, 48)   # ... but the filter's inputs of q
    assert caches[1].state.shape == (5, (4 * 6 * 10 + 3 * (24 + 2 * 2 * 10) + 3) // 4 * 4)
    ones = engine(*dirs["ones"][::2], 8)
    assert ones.cache.layer_caches[0].states == ()                             # one tap remembers nothing


def test_covering_needs():
    a, b = KVCacheNeed(2, 8, 10, keep_first=3), KVCacheNeed(2, 8, 7, keep_first=9)
    assert a.covering(b) == b.covering(a) == KVCacheNeed(2, 8, 10, keep_first=9)
    assert a.covering(KVCacheNeed(2, 8)) == KVCacheNeed(2, 8)                  # one reader sees everything
    with pytest.raises(ValueError, match="differ"):
        a.covering(KVCacheNeed(2, 12, 10))


def test_kept_pages_stay_and_the_window_s_pages_are_given_back():
    """Pages of 4, a window of 6, the first 5 keys kept: two pages at the start stay, those the window passed go, all come back at the end."""
    cm = CacheManager([KVCacheNeed(1, 4, 6, keep_first=5)], 4, 12, 2, 200, dtype=torch.float32)
    seq = cm.admit("a")
    for n in range(1, 60):
        assert cm.ensure(seq, n)
        cm.commit(seq, n)
        cm.check_invariants()
        row = cm.kv_groups[0].tables[seq.slot]
        live = {i for i in range(len(row)) if row[i]}
        need = {j // 4 for j in range(n) if n - j < 6 or j < 5}              # what position n (not fed yet) and those behind it may read
        assert need <= live and len(live) <= 2 + 3, (n, live, need)
    other = cm.admit("b")
    assert cm.ensure(other, 20)
    cm.commit(other, 20)
    cm.free(seq)
    cm.check_invariants()
    cm.free(other)
    assert cm.free_pages() == 12
    assert cm.peak_pages(cm.kv_groups[0], 200, 1) == 2 + 2 + 1 and cm.peak_pages(cm.kv_groups[0], 8, 1) == 2


# ---------------------------------------------------------------- the plain functions on inputs whose answer is known
def test_plain_mechanisms_by_hand():
    f64 = torch.float64
    t = lambda *v: torch.tensor(v, dtype=f64)                                 # noqa: E731
    assert torch.allclose(plain.one_plus_norm(t([3.0, 4.0]), t(0.0, 1.0), 0.0), t([3.0, 8.0]) / 12.5 ** 0.5)
    assert torch.allclose(plain.causal_conv(t([1.0], [2.0], [5.0]), t([10.0, 1.0])), t([1.0], [12.0], [25.0]))
    x = torch.zeros(3, 1, 4, dtype=f64)
    x[:, 0] = t(1.0, 0.0, 0.0, 2.0)
    r = plain.rotate_pairs(x, 4, 100.0)                                        # angles p and p / 10
    assert torch.allclose(r[2, 0], t(math.cos(2), math.sin(2), -2 * math.sin(0.2), 2 * math.cos(0.2)))
    assert torch.equal(plain.rotate_pairs(x, 2, 100.0)[:, :, 2:], x[:, :, 2:])
    seen = plain.visible(6, 2, 1)
    assert [[j for j in range(6) if seen[i, j]] for i in range(6)] == [[0], [0, 1], [0, 1, 2], [0, 2, 3], [0, 3, 4], [0, 4, 5]]
    assert abs(plain.capped(t(3.0), 2.0).item() - 2 * math.tanh(1.5)) < 1e-12
    # one head, one state row: S_1 = dt B x, S_2 = e^(-a dt) S_1 + dt B x
    y = plain.state_space(t([[2.0]], [[3.0]]), t([[1.0]], [[4.0]]), t([[1.0]], [[10.0]]), t([0.5], [0.25]), t(math.log(2.0)), t(7.0))
    assert torch.allclose(y.flatten(), t(1.0 + 14.0, 10 * (math.exp(-0.5) * 1.0 + 0.25 * 4 * 3) + 21.0))
    z = t([1.0, -1.0, 2.0, 0.5])
    g = (t([1.0, 2.0, 3.0, 4.0]) * z / (1 + torch.exp(-z))).flatten()
    n = plain.gated_part_norm(t([1.0, 2.0, 3.0, 4.0]), z, t(1.0, 1.0, 2.0, 1.0), 2, 0.0).flatten()
    assert torch.allclose(n, t(1.0, 1.0, 2.0, 1.0) * torch.cat([g[:2] / g[:2].pow(2).mean().sqrt(), g[2:] / g[2:].pow(2).mean().sqrt()]))
    w = {"gate": t([1.0], [1.0]), "up": t([-5.0], [0.5]), "down": t([1.0, 10.0])}
    sg = 1 / (1 + math.exp(-1.702 * 2.0))
    assert abs(plain.clamped_ff(t([3.0]), w, "", 2.0).item() - (2 * sg * (-2 + 1) + 10 * 2 * sg * (1.5 + 1))) < 1e-12
    lo = plain.clamped_ff(t([-9.0]), {"gate": t([1.0]), "up": t([0.0]), "down": t([1.0])}, "", 2.0).item()      # the gate is not clamped from below
    assert abs(lo - -9.0 / (1 + math.exp(1.702 * 9.0))) < 1e-12


def test_every_tensor_matters(dirs):
    """Zeroing any one tensor of the model changes the logits: nothing that the checkpoint holds is left unused."""
    d, cfg, page = dirs["mix"]
    c0, w = plain.load_model_dir(d)
    ids = tokens(cfg["vocab"], 30, seed=2)
    want = plain.forward_logits(c0, w, ids)
    for name in w:
        broken = dict(w)
        broken[name] = torch.zeros_like(w[name])
        assert (plain.forward_logits(c0, broken, ids) - want).abs().max() > 1e-6, name


# ---------------------------------------------------------------- each mechanism alone (one layer, or two where one reads the other's keys)
SINGLE = {
    "attention": config(32, 61, [attn(4, 2, 8, 8, 6, 2)]),
    "attention_value_rows": config(32, 61, [attn(3, 1, 12, 5, 11, 4, conv=4)]),
    "attention_odd": config(27, 53, [attn(3, 3, 7, 9, 8, 3, conv=2, rot=6)]),
    "attention_wide_window": config(32, 61, [attn(2, 1, 8, 8, 500, 4)]),
    "attention_nothing_kept": config(32, 61, [attn(2, 2, 8, 8, 5, 0)]),
    "attention_many_kept": config(32, 61, [attn(2, 2, 8, 8, 3, 20)]),
    "attention_five_taps": config(32, 61, [attn(2, 1, 16, 16, 9, 2, conv=5)]),
    "attention_all_rotated": config(32, 61, [attn(2, 1, 16, 16, 9, 2, rot=16, base=10.0)]),
    "attention_rows64": config(48, 61, [attn(4, 2, 64, 64, 33, 3, rot=20, scale=0.1)]),
    "borrowed": config(32, 61, [attn(4, 2, 8, 12, 6, 2), attn(4, 2, 8, 12, 14, 7, conv=2, cap=2.0, scale=0.7, kv_from=0)]),
    "borrowed_narrow": config(32, 61, [attn(4, 2, 8, 8, 12, 5), attn(4, 2, 8, 8, 4, 1, conv=1, kv_from=0)]),
    "mamba": config(32, 61, [mamba(4, 8, 16, 1, 1)]),
    "mamba_groups": config(32, 61, [mamba(6, 5, 9, 3, 2, conv=3)]),
    "mamba_one_tap": config(27, 53, [mamba(2, 7, 3, 2, 1, conv=1)]),
    "mamba_chunks": config(32, 61, [mamba(2, 32, 64, 2, 1)]),
    "mamba_chunks128": config(32, 61, [mamba(1, 64, 128, 1, 4)]),
    "mamba_five_taps": config(32, 61, [mamba(3, 64, 20, 1, 1, conv=5)]),
    "dense": config(40, 71, [attn(1, 1, 4, 4, 3, 1, dense(52, 0.5))], alpha=0.5),
    "dense_loose": config(40, 71, [mamba(1, 4, 3, 1, 1, mlp=dense(44, 30.0))], alpha=4.0),
}


def single_dir(tmp_path, name):
    return _perturb(write_random_model(SINGLE[name], str(tmp_path), seed=3, std=0.3, norm_init="uniform"), seed=11)


@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(tmp_path, name):
    cfg = SINGLE[name]
    d = single_dir(tmp_path, name)
    ids = tokens(cfg["vocab"], 37, seed=1)
    want = plain_logits(d, ids)
    runner = engine(d, 4, 24)
    assert err(feed(runner, "w", ids, [37]), want) < 2e-5
    assert err(feed(runner, "d", ids, [20] + [1] * 17), want) < 2e-5
    assert err(feed(runner, "p", ids, [2, 3, 2, 9, 2, 7, 5, 2, 5]), want) < 2e-5


# ---------------------------------------------------------------- the engine on the stand-in kernels (CPU)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cuts_on_cpu(dirs, name):
    d, cfg, page = dirs[name]
    check_cuts(engine(d, page, 40), d, cfg["vocab"], 2e-5)


@pytest.mark.parametrize("name", ["mix", "pages"])
def test_mixed_batches_on_cpu(dirs, name):
    d, cfg, page = dirs[name]
    check_mixed(lambda pages: engine(d, page, pages), d, cfg["vocab"], page, 2e-5)


def test_a_batch_does_not_change_its_members(dirs):
    d, cfg, page = dirs["mix"]
    runner = engine(d, page, 64)
    a, b, c = (tokens(cfg["vocab"], n, seed=n) for n in (19, 7, 30))
    alone = [feed(runner, i, ids, [len(ids)]) for i, ids in enumerate((a, b, c))]
    seqs = [runner.cache.admit(k) for k in "abc"]
    first = runner.step([StepEntry(seqs[0], a[:10], range(10)), StepEntry(seqs[1], b, range(7)), StepEntry(seqs[2], c[:1], [0])])
    second = runner.step([StepEntry(seqs[2], c[1:], range(29)), StepEntry(seqs[0], a[10:11], [0])])
    third = runner.step([StepEntry(seqs[0], a[11:], range(8))])
    got_a = torch.cat([first[:10], second[29:30], third])
    got_c = torch.cat([first[17:18], second[:29]])
    assert err(got_a, alone[0]) < 1e-5 and err(first[10:17], alone[1]) < 1e-5 and err(got_c, alone[2]) < 1e-5


def test_freed_pages_and_slots_are_taken_again(dirs):
    """A request that takes the slot and the pages another one just gave back must not see what that one left."""
    d, cfg, page = dirs["mix"]
    runner = engine(d, page, 8, max_seqs=1)
    a, b = tokens(cfg["vocab"], 26, seed=1), tokens(cfg["vocab"], 11, seed=2)
    feed(runner, "a", a, [26])
    assert err(feed(runner, "b", b, [4, 1, 1, 5]), plain_logits(d, b)) < 2e-5


def test_the_first_tokens_of_a_sequence(dirs):
    """Positions 0 .. 7: filters that reach before the start, one key, kept keys that do not all exist yet; one by one and in twos, and a
    sequence of one token."""
    for name in ("mix", "pages", "ones"):
        d, cfg, page = dirs[name]
        runner = engine(d, page, 40)
        ids = tokens(cfg["vocab"], 8, seed=9)
        want = plain_logits(d, ids)
        assert err(feed(runner, "a", ids, [1] * 8), want) < 2e-5
        assert err(feed(runner, "b", ids, [2] * 4), want) < 2e-5
        assert err(feed(runner, "c", ids[:1], [1]), want[:1]) < 2e-5


def llm_cpu(d, **kw):
    kw.setdefault("kv_cache_tokens", 512)
    return LLM(d, dtype="float32", device="cpu", ops=TorchRefOps(), **kw)


def plain_greedy(d, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(plain_logits(d, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("chunked", [False, True])
def test_generate_through_the_entry_point_on_cpu(dirs, chunked):
    d, cfg, page = dirs["mix"]
    prompts = [tokens(cfg["vocab"], n, seed=40 + n) for n in (5, 13, 22, 9, 3)]
    want = [plain_greedy(d, p, 6) for p in prompts]
    llm = llm_cpu(d, kv_block_size=page, max_num_seqs=3, chunked_prefill=chunked, max_batched_tokens=16 if chunked else 64)
    got = llm.generate(prompts, SamplingParams(max_new_tokens=6, ignore_eos=True))
    assert got == want
    assert llm.cache.free_pages() == llm.cache.num_pages and llm.cache.slots.num_free == 3


def test_preemption_recomputes_the_caches(dirs):
    d, cfg, page = dirs["pages"]
    prompts = [tokens(cfg["vocab"], n, seed=60 + n) for n in (14, 15, 13)]
    want = [plain_greedy(d, p, 8) for p in prompts]
    llm = llm_cpu(d, kv_block_size=page, kv_cache_tokens=64, max_num_seqs=3, kv_watermark=0.0)
    assert llm.generate(prompts, SamplingParams(max_new_tokens=8, ignore_eos=True)) == want
    assert llm.scheduler.preemptions > 0


def test_trace_replay_in_process(dirs, tmp_path, monkeypatch, capsys):
    from mini_inference_b200.cli import trace_run
    d, cfg, page = dirs["pages"]
    a, b = tokens(cfg["vocab"], 9, seed=1), tokens(cfg["vocab"], 6, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:5], "want": [4]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [0, 3]}, {"id": "a", "tokens": a[5:6], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[6:], "want": [2]}], "end": ["a"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    monkeypatch.setattr("mini_inference_b200.engine.factory.make_runner",
                        lambda model, *a_, **k: make_runner(model, *a_, **{**k, "ops": TorchRefOps()}))
    assert trace_run.main(["--model", d, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128", "--device", "cpu",
                           "--page-size", str(page)]) == 0
    assert [line for line in capsys.readouterr().out.split("\n") if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = plain_logits(d, a), plain_logits(d, b)
    g0 = torch.from_numpy(np.fromfile(os.path.join(tmp_path, "0.f32"), dtype="<f4").reshape(1, -1))
    g1 = torch.from_numpy(np.fromfile(os.path.join(tmp_path, "1.f32"), dtype="<f4").reshape(3, -1))
    g2 = torch.from_numpy(np.fromfile(os.path.join(tmp_path, "2.f32"), dtype="<f4").reshape(1, -1))
    assert err(g0, wa[4:5]) < 2e-5 and err(g1, torch.stack([wb[2], wb[5], wa[5]])) < 2e-5 and err(g2, wa[8:9]) < 2e-5


# ---------------------------------------------------------------- inputs made so that a fault shows
def _i32(v, device):
    return torch.tensor(v, dtype=torch.int32, device=device)


def hot_key_case(ops, device, dtype, L, hot, window, keep, page=16, rows=1, H=4, KV=2, D=24, V=24, cap=12.0):
    """L cached keys over shuffled pages, every one orthogonal to the last query except key `hot`, whose scaled score is 30 before the cap.
    The last query's weights are then known in closed form: e^(cap tanh(30 / cap)) for `hot` and 1 for every other key it sees.  Pages
    that hold only keys the window has passed are given to the null page (as the cache manager leaves them), which holds large rows.
    A key that is lost, one too many at either end, or a cap left out shows in every head."""
    g = torch.Generator().manual_seed(L * 1000 + hot)
    keys, vals = torch.randn(L, KV, D, generator=g) * 0.3, torch.randn(L, KV, V, generator=g)
    target = torch.randn(D, generator=g)
    target = target / target.norm()
    keys -= (keys @ target)[..., None] * target
    keys[hot] += 6.0 * target
    pages = -(-L // page)
    order = (torch.randperm(pages, generator=g) + 1).tolist()
    kc, vc = torch.full((pages + 1, KV, page, D), 50.0), torch.full((pages + 1, KV, page, V), 50.0)
    for j in range(L):
        kc[order[j // page], :, j % page], vc[order[j // page], :, j % page] = keys[j], vals[j]
    first = L - rows                                              # the first query's position
    table = torch.zeros(2, pages, dtype=torch.int32)
    for i in range(pages):
        if i * page < keep or (i + 1) * page > first - window + 1:
            table[1, i] = order[i]
    tiles = [(0, r) for r in range(0, rows, 64)] if rows > 1 else []
    meta = SimpleNamespace(seg_q_start=_i32([0, rows], device), seg_pos0=_i32([first], device), seg_kv_len=_i32([L], device),
                           table_rows=_i32([1], device), block_table=table.to(device), max_pages=pages, page_size=page,
                           decode_segs=_i32([0] if rows == 1 else [], device), prefill_tiles=_i32(tiles, device).view(-1, 2), tile=64, max_kv_len=L)
    q = torch.randn(rows, H, D, generator=g)
    q[-1] = 10.0 * target                                         # times the scale of 0.5: 5, times the key's 6: a score of 30
    gate = torch.randn(rows, 3 + H * V + 1, generator=g).to(dtype)
    out = ops.masked_attention(q.reshape(rows, H * D).to(device, dtype), kc.to(device, dtype), vc.to(device, dtype), meta, H, KV, D, V, 0.5, None,
                               window, False, softcap=cap, keep_first=keep, gate=gate.to(device)[:, 2:2 + H * V]).float().cpu()[-1].view(H, V)
    j = torch.arange(L)
    s = torch.zeros(L, dtype=torch.float64)
    s[hot] = 30.0 if cap is None else cap * math.tanh(30.0 / cap)
    s[~((L - 1 - j < window) | (j < keep))] = float("-inf")
    kvh = torch.arange(H) // (H // KV)
    want = torch.einsum("j,jhd->hd", torch.softmax(s, -1), vals.double()[:, kvh]) * torch.sigmoid(gate[-1, 2:2 + H * V].double()).view(H, V)
    return out, want.float()


# (L, hot, window, keep): the oldest key inside the window and the newest outside it, the last kept key and the first that is not, a
# window and kept keys that overlap, touch or leave a gap of one, edges on page borders, everything visible, one key
HOT = [(90, 53, 37, 5), (90, 52, 37, 5), (90, 4, 37, 5), (90, 5, 37, 5), (90, 0, 37, 5), (90, 89, 37, 5), (90, 26, 64, 16), (90, 25, 64, 16), (90, 15, 64, 16),
       (90, 16, 64, 17), (90, 60, 30, 60), (90, 59, 30, 60), (90, 59, 30, 59), (90, 30, 100, 4), (40, 20, 20, 19), (40, 19, 20, 19), (40, 3, 1, 0), (40, 39, 1, 0),
       (17, 0, 17, 0), (18, 0, 17, 0), (1, 0, 4, 2), (3, 0, 1, 2), (130, 64, 66, 0), (130, 63, 66, 0), (200, 70, 20, 100)]


@pytest.mark.parametrize("L,hot,window,keep", HOT)
def test_window_and_kept_edges_on_cpu(L, hot, window, keep):
    for rows in (1, min(3, L)):
        out, want = hot_key_case(TorchRefOps(), "cpu", torch.float32, L, hot, window, keep, rows=rows)
        assert (out - want).abs().max() < 1e-4 * want.abs().max() + 1e-6


def remembering_case(ops, device, dtype, cuts, H=2, V=32, N=64, G=1, taps=3):
    """A state that must remember: token 0 alone writes (its B and x are large), 300 quiet tokens follow, and the last one reads.  The
    decay is the same at every token, so what is read is known: C . B x dt e^(A dt 300) -- a lost or restarted state, a chunk's decay that
    is one token off, or a wrong slot shows.  Returns (rows of the last token before the gated norm's scale, the wanted ones)."""
    g = torch.Generator().manual_seed(5)
    T, I, C = 301, H * V, H * V + 2 * G * N
    p = torch.zeros(T, (I + C + H + 7) // 8 * 8)
    p[:, :I] = 3.0                                                # z: the gate, the same everywhere
    p[0, I:I + C] = torch.randn(C, generator=g).abs() + 0.5
    p[T - 1, 2 * I + G * N:2 * I + 2 * G * N] = torch.randn(G * N, generator=g).abs() + 0.5          # C of the last token
    p[:, I + C:I + C + H] = -5.0                                  # dt before its bias
    p = p.to(dtype)
    conv = torch.zeros(C, taps)
    conv[:, -1] = 1.0                                             # the filter passes the token itself
    dt_bias, A, Dv = torch.tensor([0.3, 0.5][:H]), torch.tensor([-0.2, -0.6][:H]), torch.zeros(H)
    norm = torch.ones(I)
    state = torch.full((2, (H * N * V + (taps - 1) * C + 3) // 4 * 4), 0.0)
    mv = lambda t: t.to(device)                                   # noqa: E731
    args = [mv(conv), torch.zeros(C, device=device), taps, mv(dt_bias), mv(A), mv(Dv), H, V, N, G, mv(norm), 1, 1e-12, mv(state)]
    at = 0
    for n in cuts:
        batch = SimpleNamespace(num_segs=1, host={"seg_q_start": [0, n], "seg_slot": [1]}, seg_q_start=_i32([0, n], device), seg_slot=_i32([1], device), token_seg=_i32([0] * n, device),
                                positions=_i32(list(range(at, at + n)), device))
        out = ops.mamba2_mix(p[at:at + n].to(device), *args, batch)
        at += n
    assert at == T
    dt = torch.nn.functional.softplus(p[0, I + C:I + C + H].double() + dt_bias.double())
    silu = lambda t: torch.nn.functional.silu(t.double())         # noqa: E731
    x0, B0 = silu(p[0, I:2 * I]).view(H, V), silu(p[0, 2 * I:2 * I + N])
    CT = silu(p[T - 1, 2 * I + N:2 * I + 2 * N])
    y = (torch.exp(A.double() * dt * 300) * dt * (B0 @ CT))[:, None] * x0
    y = (y * silu(p[T - 1, :1])).reshape(-1)
    return out[-1].float().cpu(), (y / y.pow(2).mean().sqrt()).float(), args[-1][1].float().cpu()


CUTS_301 = [[301], [300, 1], [1] * 301, [64, 64, 64, 64, 45], [2, 63, 65, 1, 1, 2, 100, 67], [299, 2]]


@pytest.mark.parametrize("cuts", CUTS_301, ids=lambda c: f"{len(c)}cuts")
def test_a_state_that_must_remember_on_cpu(cuts):
    out, want, _ = remembering_case(TorchRefOps(), "cpu", torch.float32, cuts)
    assert (out - want).abs().max() < 1e-4 * want.abs().max()


# ================================================================ on the GPU
TOL = {"float32": 1e-4, "bfloat16": 0.15}


def cuda_ops():
    from mini_inference_b200.ops import get_ops
    return get_ops("cuda:0")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cuts_on_gpu(dirs, name, dtype):
    d, cfg, page = dirs[name]
    check_cuts(engine(d, page, 40, dtype, "cuda:0"), d, cfg["vocab"], TOL[dtype])
    cuda_ops().check_errors()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "pages"])
def test_mixed_batches_on_gpu(dirs, name, dtype):
    d, cfg, page = dirs[name]
    check_mixed(lambda pages: engine(d, page, pages, dtype, "cuda:0"), d, cfg["vocab"], page, TOL[dtype])
    cuda_ops().check_errors()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone_on_gpu(tmp_path, name, dtype):
    cfg = SINGLE[name]
    d = single_dir(tmp_path, name)
    ids = tokens(cfg["vocab"], 150, seed=1)
    want = plain_logits(d, ids)
    runner = engine(d, 16, 16, dtype, "cuda:0")
    assert_close(feed(runner, "w", ids, [150]), want, TOL[dtype], "whole")
    assert_close(feed(runner, "d", ids, [110] + [1] * 40), want, TOL[dtype], "decode")
    assert_close(feed(runner, "p", ids, [2, 64, 3, 17, 2, 33, 29]), want, TOL[dtype], "portions")
    cuda_ops().check_errors()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("L,hot,window,keep", HOT + [(1500, 1363, 137, 20), (1500, 1362, 137, 20), (1500, 19, 137, 20), (1500, 20, 137, 20), (1500, 475, 1025, 3)])
def test_window_and_kept_edges_on_gpu(L, hot, window, keep, dtype):
    ops = cuda_ops()
    for D, V in ((24, 24), (64, 64), (40, 12), (128, 128)):
        for rows in (1, 3, 70):
            for splits in (None, 3):
                ops.force_splits = splits
                try:
                    out, want = hot_key_case(ops, "cuda:0", dtype, L, hot, window, keep, rows=min(rows, L), D=D, V=V)
                finally:
                    ops.force_splits = None
                assert (out - want).abs().max() < (1e-4 if dtype == torch.float32 else 2e-2) * want.abs().max() + 1e-6, (D, V, rows, splits)
    ops.check_errors()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cuts", CUTS_301, ids=lambda c: f"{len(c)}cuts")
def test_a_state_that_must_remember_on_gpu(cuts, dtype):
    ops = cuda_ops()
    for V, N in ((32, 64), (64, 128), (6, 20)):
        for chunked in (True, False):
            ops.chunked_scan = chunked
            try:
                out, want, state = remembering_case(ops, "cuda:0", dtype, cuts, V=V, N=N)
            finally:
                ops.chunked_scan = True
            assert (out - want).abs().max() < (1e-4 if dtype == torch.float32 else 2e-2) * want.abs().max(), (V, N, chunked)
            ref = remembering_case(TorchRefOps(), "cpu", dtype, [301], V=V, N=N)[2]
            assert (state - ref).abs().max() < (1e-4 if dtype == torch.float32 else 2e-3) * ref.abs().max(), (V, N, chunked)
    ops.check_errors()


@gpu
@pytest.mark.parametrize("lens,starts", [([1, 23, 6, 2], [40, 0, 100, 0]), ([300, 1, 59, 2, 130], [0, 7, 300, 3, 0]), ([1, 1, 1], [5, 0, 62]), ([700], [11])])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_kernels_against_the_stand_ins(dtype, lens, starts):
    """Every kernel the design added, alone, at sizes no model above has (odd ones too), several entries of unequal length in one launch,
    states and histories that earlier steps left, against the plain PyTorch statement of the same op."""
    ops, ref, dev = cuda_ops(), TorchRefOps(), "cuda:0"
    g = torch.Generator().manual_seed(0)
    tol = 3e-5 if dtype == torch.float32 else 2e-2
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype)      # noqa: E731
    f32 = lambda *s: torch.randn(*s, generator=g)                # noqa: E731
    close = lambda a, b, t=tol: (a.float().cpu() - b.float().cpu()).abs().max() <= t * max(1.0, b.float().abs().max().item())  # noqa: E731
    T, S = sum(lens), len(lens)
    pos = [p0 + i for p0, ln in zip(starts, lens) for i in range(ln)]
    starts_q = [sum(lens[:i]) for i in range(S + 1)]
    slots_of = random.Random(1).sample(range(1, S + 3), S)
    def batch(device):
        return SimpleNamespace(num_segs=S, host={"seg_q_start": starts_q, "seg_slot": slots_of}, seg_q_start=_i32(starts_q, device), seg_slot=_i32(slots_of, device), positions=_i32(pos, device),
                               token_seg=_i32([i for i, n in enumerate(lens) for _ in range(n)], device))
    cpu, gpu_b = batch("cpu"), batch(dev)
    for hid in (77, 192, 1030, 2052, 9000):
        x, y, w = f32(T, hid), rnd(T, hid), f32(hid)
        xa, xb = x.clone().to(dev), x.clone()
        ra, rb = ops.sum_rmsnorm(xa, y.to(dev), w.to(dev), 1.75, 1e-5, dtype), ref.sum_rmsnorm(xb, y, w, 1.75, 1e-5, dtype)
        assert close(xa, xb, 3e-5 if dtype == torch.float32 else 1e-4) and close(ra, rb) and ra.dtype == dtype
    page = 16
    cache_slots = (torch.randperm(2 * T, generator=g)[:T] + page).to(torch.int32)
    n_pages = 2 * T // page + 2
    for H, KV, D, V, taps, nf in ((6, 2, 8, 24, 4, 3), (3, 1, 7, 5, 3, 2), (4, 4, 16, 16, 2, 8), (5, 0, 24, 24, 4, 12), (4, 2, 64, 64, 1, 16), (2, 1, 10, 10, 5, 0),
                                  (32, 4, 128, 128, 4, 32), (40, 2, 128, 64, 3, 64)):
        C = H * D + KV * (D + V)
        p, bias, conv = rnd(T, (C + 11 + 7) // 8 * 8), f32(C), rnd(C, taps)
        qn, kn, inv = f32(H * D), f32(KV * D) if KV else None, torch.rand(nf, generator=g)
        state = f32(S + 3, max((taps - 1) * C, 1))
        ka, va = torch.zeros(n_pages, max(KV, 1), page, D, dtype=dtype), torch.zeros(n_pages, max(KV, 1), page, V, dtype=dtype)
        kb, vb, sa, sb = ka.to(dev), va.to(dev), state.clone(), state.to(dev)
        mv = lambda t: None if t is None else t.to(dev)          # noqa: E731
        want = ref.conv_qkv_cache(p, H, KV, D, V, bias, conv, taps, qn, kn, 1e-5, inv, sa, cpu, SimpleNamespace(slots=cache_slots, page_size=page), ka, va)
        got = ops.conv_qkv_cache(p.to(dev), H, KV, D, V, mv(bias), mv(conv), taps, mv(qn), mv(kn), 1e-5, mv(inv), sb, gpu_b,
                                 SimpleNamespace(slots=cache_slots.to(dev), page_size=page), kb, vb)
        assert close(got, want) and close(kb, ka) and close(vb, va) and close(sb, sa, 1e-6), (H, KV, D, V, taps)
    for H, V, N, G, taps, parts in ((4, 6, 10, 2, 4, 3), (3, 5, 7, 1, 3, 1), (2, 32, 64, 2, 4, 2), (4, 64, 128, 2, 3, 4), (2, 96, 64, 1, 2, 1), (1, 33, 24, 1, 1, 1), (6, 8, 200, 3, 5, 2)):
        I, C = H * V, H * V + 2 * G * N
        p = rnd(T, (I + C + H + 7) // 8 * 8)
        conv, cb, dtb, A, Dv, norm = f32(C, taps) * 0.5, f32(C) * 0.3, f32(H) - 2.0, -torch.exp(f32(H) - 1.0), f32(H), f32(I)
        state = f32(S + 3, (H * N * V + (taps - 1) * C + 3) // 4 * 4)
        sa = state.clone()
        want = ref.mamba2_mix(p, conv, cb, taps, dtb, A, Dv, H, V, N, G, norm, parts, 1e-5, sa, cpu)
        for chunked in (True, False):
            ops.chunked_scan, sb = chunked, state.to(dev)
            try:
                got = ops.mamba2_mix(p.to(dev), conv.to(dev), cb.to(dev), taps, dtb.to(dev), A.to(dev), Dv.to(dev), H, V, N, G, norm.to(dev), parts, 1e-5, sb, gpu_b)
            finally:
                ops.chunked_scan = True
            assert close(got, want) and close(sb, sa, 1e-4 if dtype == torch.float32 else 5e-3), (H, V, N, G, taps, parts, chunked)
    ops.check_errors()


def plain_judged(d, prompts, got):
    """Generated tokens judged by the plain logits: each is within a rounding's reach of the largest."""
    for p, out in zip(prompts, got):
        logits = plain_logits(d, p + out)
        for i, tok in enumerate(out):
            row = logits[len(p) + i - 1]
            assert row[tok] >= row.max() - 0.1 * row.abs().max()


@gpu
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["mix", "pages"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_generate_through_the_entry_point_on_gpu(dirs, dtype, name, graphs):
    d, cfg, page = dirs[name]
    prompts = [tokens(cfg["vocab"], n, seed=40 + n) for n in (5, 13, 22, 9, 3, 30)]
    llm = LLM(d, dtype=dtype, kv_block_size=page, kv_cache_tokens=1024, max_num_seqs=4, cuda_graphs=graphs)
    got = llm.generate(prompts, SamplingParams(max_new_tokens=12, ignore_eos=True))
    assert llm.cache.free_pages() == llm.cache.num_pages
    if graphs:
        assert llm.graphs.replays > 0
    if dtype == "float32":
        assert got == [plain_greedy(d, p, 12) for p in prompts]
    else:
        plain_judged(d, prompts, got)


@gpu
def test_long_decoding_on_gpu(dirs):
    """300 tokens generated one by one after a short prompt, through the scheduler: pages fill, the windows' pages are given back and taken
    again, the kept ones stay, and the plain implementation agrees on the whole sequence at the end."""
    d, cfg, page = dirs["pages"]
    prompt = tokens(cfg["vocab"], 11, seed=77)
    llm = LLM(d, dtype="float32", kv_block_size=page, kv_cache_tokens=512, max_num_seqs=2)
    out = llm.generate([prompt], SamplingParams(max_new_tokens=300, ignore_eos=True))[0]
    logits = plain_logits(d, prompt + out)
    picks = logits[len(prompt) - 1:-1].argmax(-1).tolist()
    assert sum(a == b for a, b in zip(picks, out)) >= 297          # a near tie may fall the other way; it does not derail the rest


@gpu
def test_trace_run_program_on_gpu(dirs, tmp_path):
    d, cfg, page = dirs["pages"]
    a = tokens(cfg["vocab"], 70, seed=5)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:64], "want": list(range(64))}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[64:], "want": list(range(6))}], "end": ["a"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        want = plain_logits(d, a)
        g0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(64, -1))
        g1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(6, -1))
        assert_close(torch.cat([g0, g1]), want, TOL[dtype])


@gpu
def test_run_engine_command_line_on_gpu(dirs, tmp_path):
    """The serving command line on a model folder of this design: the scheduler, temperature sampling and CUDA graphs."""
    d, cfg, page = dirs["mix"]
    out = tmp_path / "m.json"
    r = subprocess.run([os.path.join(ROOT, "bin", "run_engine"), "--model", d, "--dtype", "bfloat16", "-n", "5", "-c", "3", "--warmup", "1",
                        "--max-new-tokens", "9", "--prompt-len", "5:30", "--kv-tokens", "512", "--page-size", str(page), "--temperature", "0.8",
                        "--cuda-graphs", "on", "--out", str(out)], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    data = json.loads(out.read_text())
    assert data["summary"]["engine"]["architecture"] == "Fetodra"
    assert all(run["generated_tokens"] == 9 and run["error"] is None for run in data["runs"])

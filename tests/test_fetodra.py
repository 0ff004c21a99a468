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
    """float32 (tol < 1e-2): every logit within tol of the largest.  bfloat16: the root mean square of every position within tol."""
    if tol < 1e-2:
        assert err(got, want) < tol, (what, err(got, want))
        return
    per = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    assert per.max().item() < tol and per.median().item() < tol / 2, (what, per.median().item(), per.max().item())


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

"""Kofutar in the engine against the plain implementation (tests/plain/kofutar_plain.py).

Without a GPU the engine runs on the stand-in kernel namespace (tests/ref_ops.py), which exercises configuration, weights, spec, parts,
the cache manager, the batch builder, the scheduler and the entry point.  With a GPU (-m gpu) the same checks run on the CUDA kernels in
float32 and bfloat16, plus each kernel alone against the plain statement of its op."""
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
from mini_inference_b200.config import ConfigError, ExecStep, LayerSpec, ModelSpec, PartSpec, load_config, resolve
from mini_inference_b200.config.kofutar_config import KofutarConfig
from mini_inference_b200.engine.batch import StepEntry
from mini_inference_b200.engine.factory import make_runner
from mini_inference_b200.parts.base import KVCacheNeed, NormedDelta, StateNeed, build_part
from mini_inference_b200.parts.recurrent import GatedDeltaRule
from mini_inference_b200.weights import write_random_model
from tests.design_checks import Judge, assert_close, check_cuts, check_mixed, engine, err, feed, rewrite_weights, tokens
from tests.plain import kofutar_plain as plain
from tests.ref_ops import TorchRefOps

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
gpu = pytest.mark.gpu
JUDGE = Judge(plain)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def rotation(dims, base, factor=None):
    return {"base": base, "dims": dims} if factor is None else {"base": base, "dims": dims, "scaling": {"factor": factor}}


def delta(heads, kv, dim, vdim, conv=4, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def attn(heads, kv, dim, vdim, rot, scale=0.4, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, rot, scale=0.3, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                              "q_rank": q_rank, "scale": scale, "rot": rot}}


def config(width, vocab, layers, loop=None, eps=1e-5):
    out = {"architecture": "Kofutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# Small configurations that differ from one another in every size; none makes two sizes equal by accident.
CONFIGS = {
    # a span in the middle three times; two of each kind, with and without feed-forward; part of a head rotated, with and without scaling;
    # value rows of another size than key rows
    "mix": (config(44, 131, [attn(6, 2, 8, 12, rotation(4, 300.0, 2.5), mlp=dense(40)), delta(4, 2, 6, 10, conv=3), latent(3, 6, 4, 5, 14, 11, rotation(4, 90.0), mlp=dense(28)),
                             delta(6, 3, 8, 4, conv=2, mlp=dense(36)), attn(4, 4, 10, 6, rotation(10, 50.0)), latent(5, 4, 8, 7, 9, 6, rotation(8, 1e3, 4.0))],
                   loop=(1, 4, 3)), 4),
    # one head, one tap, a query latent of one, a rotation of one pair, a factor of 1, the whole model run twice
    "ones": (config(40, 97, [delta(1, 1, 24, 20, conv=1), attn(1, 1, 16, 16, rotation(2, 10.0, 1.0), mlp=dense(30)), latent(1, 8, 2, 12, 6, 1, rotation(2, 20.0))],
                    loop=(0, 3, 2), eps=1e-6), 8),
    # pages of 16 and the sizes the tensor-core kernels take (heads of 64 and 128, latent rows of 64 and 128); more than 16 latent heads;
    # a span run "once" still passes the joining product; a layer behind the span
    "pages": (config(64, 150, [attn(4, 2, 64, 64, rotation(32, 1e4, 6.0), scale=0.125, mlp=dense(72)), delta(4, 2, 32, 32, mlp=dense(24)),
                               latent(18, 16, 16, 8, 48, 24, rotation(16, 5e3), scale=0.2), attn(3, 1, 128, 128, rotation(64, 3e5), scale=0.09),
                               latent(4, 24, 32, 16, 96, 40, rotation(32, 1e5), scale=0.13, mlp=dense(36)), delta(2, 1, 64, 128, conv=3)], loop=(1, 3, 1)), 16),
}
STD = 0.25


def _spread(d, seed=7):
    """The random-weights writer leaves decays at zero, sinks and short filters small; give every one of them values, so that leaving one
    out shows, and states that remember hundreds of tokens."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda t, s: torch.randn(t.shape, generator=g) * s      # noqa: E731
    def change(name, t):
        if name.endswith(".conv"):
            return rnd(t, 0.5) + 0.3
        if name.endswith("dt_bias"):
            return rnd(t, 1.0) - 3.0
        if name.endswith("A_log"):
            return rnd(t, 0.7) - 1.0
        if name.endswith(".sink"):
            return rnd(t, 1.0) + 1.0
    JUDGE.forget(d)
    return rewrite_weights(d, plain, change)


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    out = {}
    for i, (name, (cfg, page)) in enumerate(CONFIGS.items()):
        d = str(tmp_path_factory.mktemp("kofutar_" + name))
        write_random_model(cfg, d, seed=90 + i, std=STD, norm_init="uniform")
        out[name] = (_spread(d), cfg, page)
    return out


# ---------------------------------------------------------------- configuration, registry, spec, cache needs
def test_config_reads_every_key_and_refuses_what_is_missing():
    raw = CONFIGS["mix"][0]
    assert resolve(raw).name == "Kofutar" and resolve({"architectures": ["Kofutar"]}).name == "Kofutar"
    cfg = KofutarConfig.from_dict(raw)
    assert KofutarConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.loop == (1, 4, 3) and cfg.layers[0].ff == 40 and cfg.layers[1].ff is None and cfg.norm_eps == 1e-5
    assert cfg.layers[0].mixer_dict()["rot"] == rotation(4, 300.0, 2.5) and "scaling" not in cfg.layers[4].mixer_dict()["rot"]
    assert KofutarConfig.from_dict(CONFIGS["pages"][0]).loop == (1, 3, 1)                 # a span that runs once is still a span
    bare = {k: v for k, v in raw.items() if k != "loop"}
    assert KofutarConfig.from_dict(bare).loop is None and KofutarConfig.from_dict(dict(bare, loop=None)).loop is None
    for path, msg in ((("norm",), "norm"), (("norm", "eps"), "eps"), (("width",), "width"), (("layers", 0, "mixer", "vdim"), "vdim"), (("layers", 0, "mixer", "rot", "base"), "base"),
                      (("layers", 0, "mixer", "rot", "scaling", "factor"), "factor"), (("layers", 0, "mixer", "scale"), "scale"), (("layers", 1, "mixer", "conv"), "conv"),
                      (("layers", 2, "mixer", "q_rank"), "q_rank"), (("layers", 2, "mixer", "rot"), "rot"), (("layers", 0, "mlp", "ff"), "ff"), (("loop", "times"), "times")):
        broken = json.loads(json.dumps(raw))
        node = broken
        for p in path[:-1]:
            node = node[p]
        del node[path[-1]]
        with pytest.raises(ConfigError, match=msg):
            KofutarConfig.from_dict(broken)
    for edit, msg in ((lambda c: c["layers"][0].update(type="retention"), "retention"), (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
                      (lambda c: c["layers"][1]["mixer"].update(heads=3), "kv_heads"), (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "dims"),
                      (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "dims"), (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "dims"),
                      (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "factor"), (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
                      (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe"), (lambda c: c["loop"].update(stop=9), "loop"),
                      (lambda c: c["loop"].update(stop=1), "loop"), (lambda c: c["loop"].update(times=0), "loop")):
        bad = json.loads(json.dumps(raw))
        edit(bad)
        with pytest.raises(ConfigError, match=msg):
            KofutarConfig.from_dict(bad)


def test_spec_order_and_cache_needs(dirs):
    d, cfg, page = dirs["mix"]
    _, spec = load_config(d)
    assert spec.residual == "float32" and spec.join_name == "loop.in"
    assert [s.layer for s in spec.order] == [0] + [1, 2, 3] * 3 + [4, 5]
    assert [i for i, s in enumerate(spec.order) if s.join_embedding] == [1, 4, 7]         # before every pass, the first too
    assert [layer.block for layer in spec.layers] == ["sandwich", "sandwich_mixer", "sandwich", "sandwich", "sandwich_mixer", "sandwich_mixer"]
    assert spec.layers[5].part("position").get("factor") == 4.0 and spec.layers[2].part("position").get("factor") == 1.0
    runner = engine(d, page, 8)
    caches = runner.cache.layer_caches
    needs = {g.need: len(g.steps) for g in runner.cache.kv_groups}
    # every pass of the span has pages and states of its own
    assert needs == {KVCacheNeed(2, 8, value_dim=12): 1, KVCacheNeed(1, 14 + 4, planes=1): 3, KVCacheNeed(4, 10, value_dim=6): 1, KVCacheNeed(1, 9 + 8, planes=1): 1}
    C = 2 * 2 * 6 + 4 * 10
    assert caches[1].state.shape == (5, 4 * 6 * 10 + 3 * C) and len({caches[i].state.data_ptr() for i in (1, 4, 7)}) == 3
    ones = engine(*dirs["ones"][::2], 8)
    assert ones.cache.layer_caches[0].state.shape == (5, 24 * 20)                          # one tap remembers no inputs
    _, once = load_config(dirs["pages"][0])
    assert [s.join_embedding for s in once.order] == [False, True, False, False, False, False]


def test_a_join_needs_its_weight_and_a_float32_stream():
    norm = PartSpec.of("stream_layernorm", size=8, eps=1e-5)
    layer = LayerSpec.of("sandwich_mixer", {}, mixer=PartSpec.of("gated_delta"), norm1=norm, norm1b=norm, position=PartSpec.of("none"))
    kw = dict(hidden_size=8, vocab_size=9, layers=(layer,), order=(ExecStep(0, join_embedding=True),), final_norm=norm, embedding_name="embed",
              final_norm_name="f", lm_head_name="head", max_position=64)
    for extra in (dict(residual="float32"), dict(join_name="w")):
        with pytest.raises(ValueError, match="joins"):
            ModelSpec(**kw, **extra)
    with pytest.raises(ValueError, match="both sides"):
        build_part("block", PartSpec.of("sandwich_mixer"), dict(mixer=None, norm1=build_part("norm", PartSpec.of("stream_rmsnorm", size=8, eps=1e-5)),
                                                               norm1b=build_part("norm", norm), position=None))
    with pytest.raises(ValueError, match="gate"):
        build_part("mixer", PartSpec.of("latent_attention", hidden_size=8, num_heads=1, nope_dim=2, rot_dim=2, value_dim=2, kv_rank=2, scale=1.0,
                                        latent_norm_eps=1e-5, gate="rows"))


def test_the_count_of_operations_knows_the_join(dirs):
    """step_flops: 2 per weight element and row for every layer run, the joined halves included (the embedded half once)."""
    d, cfg, page = dirs["ones"]
    model = engine(d, page, 8).model
    runs = model.step_flops(10, 0, 0) - 10 * 8 * (24 * 20) * 2
    matrices = sum(2 * 10 * v.numel() for s in model.spec.order for part in model._parts_of(model.blocks[s.layer]) for v in vars(part).values()
                   if isinstance(v, torch.Tensor) and v.dim() == 2)
    per_join = 2 * 10 * 40 * 40
    latent_extra = 2 * 2 * 10 * 1 * 6 * (8 + 12)                  # the absorbed projections of the latent layer, twice
    assert runs == matrices + 2 * per_join + per_join + latent_extra


# ---------------------------------------------------------------- the plain functions on inputs whose answer is known
def test_plain_mechanisms_by_hand():
    f64 = torch.float64
    t = lambda *v: torch.tensor(v, dtype=f64)                                 # noqa: E731
    assert torch.allclose(plain.layer_norm(t(1.0, 3.0, 8.0), t(1.0, 2.0, 0.5), 0.0), t(-3.0, -2.0, 2.0) / (26 / 3) ** 0.5)
    assert torch.allclose(plain.layer_norm(t(1001.0, 1003.0, 1008.0), t(1.0, 2.0, 0.5), 0.0), t(-3.0, -2.0, 2.0) / (26 / 3) ** 0.5)
    assert torch.allclose(plain.rms_norm(t(3.0, 4.0), t(1.0, 2.0), 0.0), t(3.0, 8.0) / 12.5 ** 0.5)
    x = torch.zeros(4, 1, 5, dtype=f64)
    x[:, 0] = t(1.0, 0.0, 0.0, 2.0, 7.0)                                       # pairs (0, 2) and (1, 3); the last coordinate passes
    r = plain.rotate_half(x, 4, 100.0, 2.0)                                    # angles p / 2 and p / 20
    assert torch.allclose(r[3, 0], t(math.cos(1.5), -2 * math.sin(0.15), math.sin(1.5), 2 * math.cos(0.15), 7.0))
    assert torch.allclose(plain.causal_conv(t([1.0], [2.0], [5.0]), t([10.0, 1.0])), t([1.0], [12.0], [25.0]))
    assert torch.allclose(plain.unit(t(3.0, 4.0)), t(0.6, 0.8), atol=1e-7)
    assert abs(plain.unit(t(0.0, 1e-3), 1e-6)[1].item() - 1e-3 / math.sqrt(2e-6)) < 1e-12
    assert abs(plain.decay(t(0.7), t(math.log(2.0)), t(-0.2)).item() - math.exp(-2.0 * math.log1p(math.exp(0.5)))) < 1e-12
    # one head, one state row: S = 0.5 * 0 + k (b v) = 0.6; then S = 0.25 * 0.6 = 0.15, u = 0.5 (3 - 0.15 * 2) = 1.35, S = 0.15 + 2 * 1.35; reads q S
    o = plain.delta_scan(t([[5.0]], [[10.0]]), t([[1.0]], [[2.0]]), t([[2.0]], [[3.0]]), t([0.3], [0.5]), t([0.5], [0.25]))
    assert torch.allclose(o.flatten(), t(5 * 0.6, 10 * (0.15 + 2.7)))
    # two keys with scores 0 and ln 3, a sink of ln 4: weights 1/8, 3/8
    q, k, v = t([[0.0]], [[1.0]]), t([[0.0]], [[math.log(3.0)]]), t([[8.0]], [[16.0]])
    assert torch.allclose(plain.attend(q, k, v, 1.0, t(math.log(4.0)))[1].flatten(), t(8 / 8 + 16 * 3 / 8))
    assert torch.allclose(plain.attend(q, k, v, 1.0)[1].flatten(), t(8 / 4 + 16 * 3 / 4))
    g = 0.5 * 1.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * (1.5 + 0.044715 * 1.5 ** 3)))
    assert abs(plain.dense_ff(t([1.5]), {"gate": t([1.0]), "up": t([2.0]), "down": t([10.0])}, "").item() - 10 * g * 3.0) < 1e-12
    assert plain.layer_runs(CONFIGS["mix"][0]) == [(0, False)] + [(1, True), (2, False), (3, False)] * 3 + [(4, False), (5, False)]


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


# ---------------------------------------------------------------- each mechanism alone (one layer)
SINGLE = {
    "delta": config(32, 61, [delta(4, 2, 8, 8)]),
    "delta_odd": config(27, 53, [delta(6, 2, 7, 5, conv=3)]),                  # value columns that are no multiple of four
    "delta_own_keys": config(32, 61, [delta(3, 3, 12, 20, conv=2)]),
    "delta_one_tap": config(32, 61, [delta(2, 1, 16, 4, conv=1)]),
    "delta_six_taps": config(32, 61, [delta(2, 1, 10, 12, conv=6)]),
    "delta_wide": config(32, 61, [delta(2, 2, 96, 132)]),
    "delta_rows128": config(32, 61, [delta(2, 1, 128, 128)]),
    "attention": config(32, 61, [attn(4, 2, 8, 8, rotation(4, 100.0))]),
    "attention_all_rotated": config(32, 61, [attn(2, 1, 16, 16, rotation(16, 10.0, 3.0))]),
    "attention_none_rotated": config(32, 61, [attn(2, 1, 16, 16, rotation(0, 10.0))]),
    "attention_odd": config(27, 53, [attn(3, 3, 7, 9, rotation(6, 40.0))]),
    "attention_rows112": config(48, 61, [attn(6, 3, 112, 112, rotation(40, 1e4, 3.0), scale=0.1)]),
    "attention_rows64": config(48, 61, [attn(4, 2, 64, 64, rotation(20, 1e4), scale=0.1)]),
    "latent": config(32, 61, [latent(4, 8, 4, 8, 12, 10, rotation(4, 100.0))]),
    "latent_odd": config(27, 53, [latent(3, 7, 6, 5, 9, 11, rotation(6, 30.0, 2.0))]),
    "latent_part_rotated": config(32, 61, [latent(2, 8, 8, 4, 12, 6, rotation(4, 30.0))]),
    "latent_rows64": config(32, 61, [latent(5, 16, 16, 12, 48, 8, rotation(16, 1e3))]),
    "latent_many_heads": config(32, 61, [latent(20, 16, 32, 4, 96, 8, rotation(32, 1e3))]),
    "dense": config(40, 71, [delta(1, 1, 4, 4, mlp=dense(52))]),
    "looped": config(36, 71, [latent(2, 6, 4, 6, 8, 5, rotation(4, 50.0), mlp=dense(20))], loop=(0, 1, 4)),
    "looped_delta": config(36, 71, [delta(2, 1, 6, 8, mlp=dense(20))], loop=(0, 1, 3)),
}


def single_dir(tmp_path, name):
    return _spread(write_random_model(SINGLE[name], str(tmp_path), seed=3, std=0.3, norm_init="uniform"), seed=11)


@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(tmp_path, name):
    cfg = SINGLE[name]
    d = single_dir(tmp_path, name)
    ids = tokens(cfg["vocab"], 37, seed=1)
    want = JUDGE.logits(d, ids)
    runner = engine(d, 4, 24)
    assert err(feed(runner, "w", ids, [37]), want) < 2e-5
    assert err(feed(runner, "d", ids, [20] + [1] * 17), want) < 2e-5
    assert err(feed(runner, "p", ids, [2, 3, 2, 9, 2, 7, 5, 2, 5]), want) < 2e-5


# ---------------------------------------------------------------- the engine on the stand-in kernels (CPU)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cuts_on_cpu(dirs, name):
    d, cfg, page = dirs[name]
    check_cuts(engine(d, page, 40), JUDGE, d, cfg["vocab"], 2e-5)


@pytest.mark.parametrize("name", ["mix", "pages"])
def test_mixed_batches_on_cpu(dirs, name):
    d, cfg, page = dirs[name]
    check_mixed(lambda pages: engine(d, page, pages), JUDGE, d, cfg["vocab"], page, 2e-5)


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
    assert err(feed(runner, "b", b, [4, 1, 1, 5]), JUDGE.logits(d, b)) < 2e-5


def test_the_first_tokens_of_a_sequence(dirs):
    """Positions 0 .. 7: filters that reach before the start, one key beside the sink; one by one and in twos, and a sequence of one token."""
    for name in ("mix", "pages", "ones"):
        d, cfg, page = dirs[name]
        runner = engine(d, page, 40)
        ids = tokens(cfg["vocab"], 8, seed=9)
        want = JUDGE.logits(d, ids)
        assert err(feed(runner, "a", ids, [1] * 8), want) < 2e-5
        assert err(feed(runner, "b", ids, [2] * 4), want) < 2e-5
        assert err(feed(runner, "c", ids[:1], [1]), want[:1]) < 2e-5


def test_a_left_out_request_goes_on_where_it_was(dirs):
    """A request that sits out steps in which others decode keeps its state, its ring of inputs and its pages."""
    d, cfg, page = dirs["mix"]
    runner = engine(d, page, 64)
    a, b = tokens(cfg["vocab"], 14, seed=21), tokens(cfg["vocab"], 20, seed=22)
    sa, sb = runner.cache.admit("a"), runner.cache.admit("b")
    got = [runner.step([StepEntry(sa, a[:5], range(5))])]
    for i in range(20):
        runner.step([StepEntry(sb, b[i:i + 1], [0])])
    got.append(runner.step([StepEntry(sa, a[5:6], [0])]))
    got.append(runner.step([StepEntry(sa, a[6:], range(8))]))
    assert err(torch.cat(got), JUDGE.logits(d, a)) < 2e-5


def llm_cpu(d, **kw):
    kw.setdefault("kv_cache_tokens", 512)
    return LLM(d, dtype="float32", device="cpu", ops=TorchRefOps(), **kw)


@pytest.mark.parametrize("chunked", [False, True])
def test_generate_through_the_entry_point_on_cpu(dirs, chunked):
    d, cfg, page = dirs["mix"]
    prompts = [tokens(cfg["vocab"], n, seed=40 + n) for n in (5, 13, 22, 9, 3)]
    want = [JUDGE.greedy(d, p, 6) for p in prompts]
    llm = llm_cpu(d, kv_block_size=page, max_num_seqs=3, chunked_prefill=chunked, max_batched_tokens=16 if chunked else 64)
    got = llm.generate(prompts, SamplingParams(max_new_tokens=6, ignore_eos=True))
    assert got == want
    assert llm.cache.free_pages() == llm.cache.num_pages and llm.cache.slots.num_free == 3


def test_preemption_recomputes_the_caches(dirs):
    d, cfg, page = dirs["pages"]
    prompts = [tokens(cfg["vocab"], n, seed=60 + n) for n in (14, 15, 13)]
    want = [JUDGE.greedy(d, p, 8) for p in prompts]
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
    wa, wb = JUDGE.logits(d, a), JUDGE.logits(d, b)
    g0 = torch.from_numpy(np.fromfile(os.path.join(tmp_path, "0.f32"), dtype="<f4").reshape(1, -1))
    g1 = torch.from_numpy(np.fromfile(os.path.join(tmp_path, "1.f32"), dtype="<f4").reshape(3, -1))
    g2 = torch.from_numpy(np.fromfile(os.path.join(tmp_path, "2.f32"), dtype="<f4").reshape(1, -1))
    assert err(g0, wa[4:5]) < 2e-5 and err(g1, torch.stack([wb[2], wb[5], wa[5]])) < 2e-5 and err(g2, wa[8:9]) < 2e-5


# ---------------------------------------------------------------- inputs made so that a fault shows
def _i32(v, device):
    return torch.tensor(v, dtype=torch.int32, device=device)


def hot_key_case(ops, device, dtype, L, hot, kind, rows=1, page=16, H=4, KV=2, D=24, V=24):
    """L cached keys over shuffled pages, every one orthogonal to the last query except key `hot`, whose scaled score is 8.  The last
    query's weights are then known in closed form: e^8 for `hot`, 1 for every other key and, for the latent kernels, e^(sink_h) for a
    sink of about 7.5 beside it.  A far key that is lost, one key too many and a sink left out, scaled or counted twice show in every
    head.  kind "latent": KV is 1 and the first V entries of a key row are its values."""
    g = torch.Generator().manual_seed(L * 1000 + hot)
    lat = kind == "latent"
    KV = 1 if lat else KV
    keys = torch.randn(L, KV, D, generator=g) * 0.3
    target = torch.randn(D, generator=g)
    target = target / target.norm()
    keys -= (keys @ target)[..., None] * target
    keys[hot] += 4.0 * target
    keys = keys.to(dtype).float()
    vals = keys[..., :V] if lat else torch.randn(L, KV, V, generator=g).to(dtype).float()
    pages = -(-L // page)
    order = (torch.randperm(pages, generator=g) + 1).tolist()
    kc, vc = torch.full((pages + 1, KV, page, D), 30.0), torch.full((pages + 1, KV, page, V), 30.0)
    for j in range(L):
        kc[order[j // page], :, j % page], vc[order[j // page], :, j % page] = keys[j], vals[j]
    table = torch.zeros(2, pages, dtype=torch.int32)
    table[1] = torch.tensor(order)
    tiles = [(0, r) for r in range(0, rows, 64)] if rows > 1 else []
    meta = SimpleNamespace(seg_q_start=_i32([0, rows], device), seg_pos0=_i32([L - rows], device), seg_kv_len=_i32([L], device),
                           table_rows=_i32([1], device), block_table=table.to(device), max_pages=pages, page_size=page,
                           decode_segs=_i32([0] if rows == 1 else [], device), prefill_tiles=_i32(tiles, device).view(-1, 2), tile=64, max_kv_len=L)
    q = torch.randn(rows, H, D, generator=g)
    q[-1] = 4.0 * target                                          # times the scale of 0.5: 2, times the key's 4: a score of 8
    q = q.to(dtype)
    sink = torch.linspace(7.0, 8.0, H) if lat else None
    if lat:
        out = ops.latent_attention(q.to(device), kc.to(device, dtype), meta, H, V, D - V, 0.5, sink_values=sink.to(device))[:, -1].float().cpu()
    else:
        out = ops.masked_attention(q.reshape(rows, H * D).to(device), kc.to(device, dtype), vc.to(device, dtype), meta, H, KV, D, V, 0.5, None, None,
                                   False).float().cpu()[-1].view(H, V)
    kvh = torch.arange(H) // (H // KV)
    s = torch.einsum("hd,jhd->hj", q[-1].double(), keys.double()[:, kvh]) * 0.5
    if lat:
        s = torch.cat([s, sink.double()[:, None]], dim=1)
    want = torch.einsum("hj,jhd->hd", torch.softmax(s, -1)[:, :L], vals.double()[:, kvh])
    assert abs(s[0, hot].item() - 8.0) < 0.1
    return out, want.float()


HOT = [(90, 0), (90, 89), (90, 15), (90, 16), (90, 63), (90, 64), (40, 31), (40, 32), (17, 16), (1, 0), (130, 1), (200, 127), (200, 128)]


@pytest.mark.parametrize("kind", ["grouped", "latent"])
@pytest.mark.parametrize("L,hot", HOT)
def test_far_keys_and_the_sink_on_cpu(L, hot, kind):
    for rows in (1, min(3, L)):
        for V in (24, 17):
            out, want = hot_key_case(TorchRefOps(), "cpu", torch.float32, L, hot, kind, rows=rows, V=V)
            assert (out - want).abs().max() < 1e-4 * want.abs().max() + 1e-6


def chunk_lists(lens, device):
    lists = GatedDeltaRule.step_arrays(SimpleNamespace(lens=lens))
    return torch.from_numpy(lists["chunks"]).to(device), torch.from_numpy(lists["first"]).to(device)


def test_chunk_lists():
    a, first = chunk_lists([1, 130, 64, 2], "cpu")
    assert a.tolist() == [[0, 0], [1, 0], [1, 64], [1, 128], [2, 0], [3, 0]] and first.tolist() == [0, 1, 4, 5]
    a, first = chunk_lists([1, 1, 1], "cpu")                       # a decode step needs none (and their number depends on the lengths alone)
    assert a.shape == (0, 2) and first.shape == (0,)


def remembering_case(ops, device, dtype, cuts, H=4, KV=2, D=16, V=12, taps=3, T=301):
    """A state that must remember: token 0 alone writes (beta near 1 at it, next to nothing behind it), 300 quiet tokens with keys
    orthogonal to the first follow, and the last one asks with the first one's key.  What is read is known: f^300 D^-1/2 beta_0 v_0 -- a
    lost or restarted state, a decay that is one token off or a wrong slot shows.  Returns (the last token's rows, the wanted ones, the slot)."""
    g = torch.Generator().manual_seed(5)
    C = 2 * KV * D + H * V
    p = torch.zeros(T, (C + H * V + 2 * H + 7) // 8 * 8)
    q, k = p[:, :KV * D].view(T, KV, D), p[:, KV * D:2 * KV * D].view(T, KV, D)
    half = D // 2                                                  # the first key lives in the first half of the coordinates, the others' in the second
    k[0, :, :half] = torch.rand(KV, half, generator=g) + 0.5
    k[1:, :, half:] = torch.rand(T - 1, KV, D - half, generator=g) + 0.5
    q[T - 1] = k[0]
    p[:, 2 * KV * D:C] = torch.randn(T, H * V, generator=g)
    p[:, C:C + H * V] = 2.0                                        # the gate, the same everywhere
    p[:, C + H * V:C + H * V + H] = -30.0
    p[0, C + H * V:C + H * V + H] = 3.0
    p[:, C + H * V + H:C + H * V + 2 * H] = -5.0
    p = p.to(dtype)
    conv = torch.zeros(C, taps)
    conv[:, -1] = 1.0                                              # the filter passes the token itself
    rate, dt_bias = torch.linspace(0.2, 0.9, H), torch.linspace(0.3, -0.2, H)
    norm = torch.linspace(0.5, 1.5, V)
    state = torch.zeros(2, (H * D * V + (taps * C if taps > 1 else 0) + 3) // 4 * 4)
    st = state.to(device)
    at = 0
    for n in cuts:
        batch = SimpleNamespace(num_segs=1, host={"seg_q_start": [0, n], "seg_slot": [1]}, seg_q_start=_i32([0, n], device), seg_slot=_i32([1], device),
                                token_seg=_i32([0] * n, device), positions=_i32(list(range(at, at + n)), device))
        out = ops.gated_delta_mix(p[at:at + n].to(device), conv.to(device), taps, rate.to(device), dt_bias.to(device), H, KV, D, V, 1e-6, norm.to(device), 1e-12,
                                  st, batch, chunks=chunk_lists([n], device) if n > 1 else None)
        at += n
    assert at == T
    silu = torch.nn.functional.silu
    unit = lambda v: v / torch.sqrt(v.pow(2).sum(-1, keepdim=True) + 1e-6)      # noqa: E731
    ku = unit(silu(p[0, KV * D:2 * KV * D].double().view(KV, D))).repeat_interleave(H // KV, dim=0)
    v0 = silu(p[0, 2 * KV * D:C].double()).view(H, V)
    f = torch.exp(-rate.double() * torch.nn.functional.softplus(p[0, C + H * V + H:C + H * V + 2 * H].double() + dt_bias.double()))
    S = ku[:, :, None] * (torch.sigmoid(p[0, C + H * V:C + H * V + H].double())[:, None] * v0)[:, None, :] * (f ** 300)[:, None, None]
    o = torch.einsum("hdv,hd->hv", S, ku) * D ** -0.5
    want = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + 1e-12) * norm.double() * silu(p[T - 1, C:C + H * V].double()).view(H, V)
    return out[-1].float().cpu().view(H, V), want.float(), st[1].float().cpu()[:H * D * V].view(H, D, V), S.float()


CUTS_301 = [[301], [300, 1], [1] * 301, [64, 64, 64, 64, 45], [2, 63, 65, 1, 1, 2, 100, 67], [299, 2]]


@pytest.mark.parametrize("cuts", CUTS_301, ids=lambda c: f"{len(c)}cuts")
def test_a_state_that_must_remember_on_cpu(cuts):
    out, want, state, S = remembering_case(TorchRefOps(), "cpu", torch.float32, cuts)
    assert (out - want).abs().max() < 1e-4 * want.abs().max() and (state - S).abs().max() < 1e-4 * S.abs().max()


def test_the_variance_is_taken_from_the_mean():
    """A row with a large common part: sums of raw squares would lose what the norm divides by."""
    g = torch.Generator().manual_seed(1)
    x = torch.randn(3, 64, generator=g) + 3000.0
    w = torch.rand(64, generator=g) + 0.5
    got = TorchRefOps().stream_layernorm(x.clone(), None, None, w, 1e-6, None, torch.float32)
    assert torch.allclose(got.double(), plain.layer_norm(x.double(), w.double(), 1e-6), atol=2e-3)


# ================================================================ on the GPU
TOL = {"float32": 1e-4, "bfloat16": 0.2}        # bfloat16: narrow rows and a dozen layer runs between norms pass a rounding on undamped; the stand-ins show the same


def cuda_ops():
    from mini_inference_b200.ops import get_ops
    return get_ops("cuda:0")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cuts_on_gpu(dirs, name, dtype):
    d, cfg, page = dirs[name]
    check_cuts(engine(d, page, 40, dtype, "cuda:0"), JUDGE, d, cfg["vocab"], TOL[dtype])
    cuda_ops().check_errors()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "pages"])
def test_mixed_batches_on_gpu(dirs, name, dtype):
    d, cfg, page = dirs[name]
    check_mixed(lambda pages: engine(d, page, pages, dtype, "cuda:0"), JUDGE, d, cfg["vocab"], page, TOL[dtype])
    cuda_ops().check_errors()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone_on_gpu(tmp_path, name, dtype):
    cfg = SINGLE[name]
    d = single_dir(tmp_path, name)
    ids = tokens(cfg["vocab"], 150, seed=1)
    want = JUDGE.logits(d, ids)
    runner = engine(d, 16, 16, dtype, "cuda:0")
    assert_close(feed(runner, "w", ids, [150]), want, TOL[dtype], "whole")
    assert_close(feed(runner, "d", ids, [110] + [1] * 40), want, TOL[dtype], "decode")
    assert_close(feed(runner, "p", ids, [2, 64, 3, 17, 2, 33, 29]), want, TOL[dtype], "portions")
    cuda_ops().check_errors()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("L,hot", HOT + [(1500, 3), (1500, 700), (1500, 1499), (1100, 1023)])
def test_far_keys_and_the_sink_on_gpu(L, hot, dtype):
    ops = cuda_ops()
    for kind, H, D, V in (("grouped", 4, 24, 24), ("grouped", 4, 64, 64), ("grouped", 6, 112, 112), ("grouped", 4, 40, 12), ("grouped", 4, 128, 128),
                          ("latent", 4, 88, 72), ("latent", 5, 64, 48), ("latent", 20, 128, 96), ("latent", 3, 24, 17)):
        for rows in (1, 3, 70):
            for splits in (None, 3):
                ops.force_splits = splits
                try:
                    out, want = hot_key_case(ops, "cuda:0", dtype, L, hot, kind, rows=min(rows, L), H=H, D=D, V=V)
                finally:
                    ops.force_splits = None
                assert (out - want).abs().max() < (1e-4 if dtype == torch.float32 else 2e-2) * want.abs().max() + 1e-6, (kind, H, D, V, rows, splits)
    ops.check_errors()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cuts", CUTS_301, ids=lambda c: f"{len(c)}cuts")
def test_a_state_that_must_remember_on_gpu(cuts, dtype):
    ops = cuda_ops()
    for H, KV, D, V, taps in ((4, 2, 16, 12, 3), (2, 1, 128, 128, 4), (4, 4, 64, 32, 1), (3, 1, 20, 7, 2), (2, 2, 64, 128, 4), (3, 1, 64, 64, 2), (2, 1, 128, 64, 3)):
        for fused in (True, False):                                # decode steps in one kernel; prompts in chunks where the sizes have the form
            ops.fused_delta_step = ops.chunked_scan = fused
            try:
                out, want, state, S = remembering_case(ops, "cuda:0", dtype, cuts, H, KV, D, V, taps)
            finally:
                ops.fused_delta_step = ops.chunked_scan = True
            assert (out - want).abs().max() < (1e-4 if dtype == torch.float32 else 2e-2) * want.abs().max(), (H, KV, D, V, taps, fused)
            assert (state - S).abs().max() < (1e-4 if dtype == torch.float32 else 2e-3) * S.abs().max(), (H, KV, D, V, taps, fused)
    ops.check_errors()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_norm_kernel_against_the_stand_in(dtype):
    ops, ref, dev = cuda_ops(), TorchRefOps(), "cuda:0"
    g = torch.Generator().manual_seed(2)
    f32 = lambda *s: torch.randn(*s, generator=g)                # noqa: E731
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    rows = torch.tensor([4, 0, 4], dtype=torch.int32)
    for T, hid in ((7, 77), (5, 64), (9, 192), (6, 1030), (5, 2052), (6, 4096), (5, 9000)):
        x, y, pre, w, wy = f32(T, hid) * 2 + 5, (f32(T, hid) * 3 - 1).to(dtype), f32(T, hid), f32(hid), f32(hid)
        mv = lambda t: None if t is None else t.to(dev)          # noqa: E731
        for use_y, use_pre, use_w, use_rows in ((1, 0, 1, 0), (0, 0, 1, 0), (0, 1, 1, 0), (1, 1, 1, 0), (1, 0, 0, 0), (1, 0, 1, 1), (0, 0, 1, 1)):
            xa, xb = x.clone(), x.clone().to(dev)
            args = lambda mv: (mv(pre) if use_pre else None, mv(w) if use_w else None, 1e-5, mv(rows) if use_rows else None, dtype)      # noqa: E731
            want = ref.stream_layernorm(xa, NormedDelta(y, wy, 1e-4) if use_y else None, *args(lambda t: t))
            got = ops.stream_layernorm(xb, NormedDelta(mv(y), mv(wy), 1e-4) if use_y else None, *args(mv))
            assert got.dtype == dtype and (got.float().cpu() - want.float()).abs().max() <= tol * max(1.0, want.float().abs().max().item()), (T, hid, use_y, use_pre, use_w, use_rows)
            assert (xb.cpu() - xa).abs().max() <= 2e-5 * max(1.0, xa.abs().max().item())
            assert torch.equal(xb.cpu(), x) == bool(use_rows or not use_w or not (use_y or use_pre))     # who leaves the stream as it is
    # a large common part costs no digits of the deviation
    x, w = f32(4, 2048) + 3000.0, torch.ones(2048)
    got = ops.stream_layernorm(x.to(dev), None, None, w.to(dev), 1e-6, None, dtype).float().cpu()
    assert (got.double() - plain.layer_norm(x.double(), w.double(), 1e-6)).abs().max() < (2e-3 if dtype == torch.float32 else 3e-2)


@gpu
@pytest.mark.parametrize("lens,starts", [([1, 23, 6, 2], [40, 0, 100, 0]), ([300, 1, 59, 2, 130], [0, 7, 300, 3, 0]), ([1, 1, 1], [5, 0, 62]), ([1100], [11])])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_kernels_against_the_stand_ins(dtype, lens, starts):
    """Every kernel the design added or widened, alone, at sizes no model above has (odd ones too), several entries of unequal length in
    one launch, states and rings that earlier steps left, against the plain PyTorch statement of the same op."""
    ops, ref, dev = cuda_ops(), TorchRefOps(), "cuda:0"
    g = torch.Generator().manual_seed(0)
    tol = 3e-5 if dtype == torch.float32 else 2e-2
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype)      # noqa: E731
    f32 = lambda *s: torch.randn(*s, generator=g)                # noqa: E731
    mv = lambda t: None if t is None else t.to(dev)              # noqa: E731
    close = lambda a, b, t=tol: (a.float().cpu() - b.float().cpu()).abs().max() <= t * max(1.0, b.float().abs().max().item())  # noqa: E731
    T, S = sum(lens), len(lens)
    pos = [p0 + i for p0, ln in zip(starts, lens) for i in range(ln)]
    starts_q = [sum(lens[:i]) for i in range(S + 1)]
    slots_of = random.Random(1).sample(range(1, S + 3), S)
    def batch(device):
        return SimpleNamespace(num_segs=S, host={"seg_q_start": starts_q, "seg_slot": slots_of}, seg_q_start=_i32(starts_q, device), seg_slot=_i32(slots_of, device),
                               positions=_i32(pos, device), token_seg=_i32([i for i, n in enumerate(lens) for _ in range(n)], device))
    cpu, gpu_b = batch("cpu"), batch(dev)
    for n in (8, 13, 200, 1032):
        r, gate = rnd(T, n), rnd(T, n + 24)
        for off in (0, 5, 8):
            assert close(ops.sigmoid_gate(r.clone().to(dev), gate.to(dev)[:, off:off + n]), ref.sigmoid_gate(r.clone(), gate[:, off:off + n]))
    page = 16
    cache_slots = (torch.randperm(2 * T, generator=g)[:T] + page).to(torch.int32)
    n_pages = 2 * T // page + 2
    ca, cg = SimpleNamespace(slots=cache_slots, positions=cpu.positions, page_size=page), SimpleNamespace(slots=cache_slots.to(dev), positions=gpu_b.positions, page_size=page)
    for H, KV, D, V, half in ((6, 2, 8, 24, 3), (3, 1, 7, 5, 3), (4, 4, 16, 16, 8), (4, 2, 80, 80, 20), (2, 1, 33, 33, 0), (8, 2, 128, 128, 32), (1, 1, 256, 40, 128)):
        p, qw, kw, inv = rnd(T, (H + KV) * D + KV * V), f32(D), f32(D), torch.rand(half, generator=g)
        ka, va = torch.zeros(n_pages, KV, page, D, dtype=dtype), torch.zeros(n_pages, KV, page, V, dtype=dtype)
        kb, vb, pb = ka.to(dev), va.to(dev), p.to(dev)
        want = ref.unit_qk_cache(p, H, KV, D, V, 1e-5, None, None, ca, ka, va, q_weight=qw, k_weight=kw, inv_freq=inv)
        got = ops.unit_qk_cache(pb, H, KV, D, V, 1e-5, None, None, cg, kb, vb, q_weight=qw.to(dev), k_weight=kw.to(dev), inv_freq=inv.to(dev))
        assert close(got, want) and close(kb, ka) and close(vb, va), (H, KV, D, V, half)
    for H, D, R, C, nf, q_rank in ((3, 6, 4, 10, 2, 9), (2, 5, 8, 64, 3, 16), (4, 16, 32, 96, 16, 24), (1, 4, 2, 7, 1, 1)):
        for half in (False, True):
            p, q_abs, qp, nw, inv = rnd(T, q_rank + C + R + 11), rnd(H, T, C), rnd(T, H * (D + R)), f32(C), torch.rand(nf, generator=g)
            pa = torch.zeros(n_pages, 1, page, C + R, dtype=dtype)
            pb = pa.to(dev)
            want = ref.latent_prepare(p, q_abs, H, D, R, C, nw, 1e-5, inv, ca, pa, q_rows=qp, dkv_col=q_rank, half_pairs=half)
            got = ops.latent_prepare(mv(p), mv(q_abs), H, D, R, C, mv(nw), 1e-5, mv(inv), cg, pb, q_rows=mv(qp), dkv_col=q_rank, half_pairs=half)
            assert close(got, want) and close(pb, pa), (H, D, R, C, nf, half)
    for H, KV, D, V, taps in ((4, 2, 6, 8, 3), (3, 1, 7, 5, 2), (2, 2, 32, 64, 4), (6, 2, 64, 36, 1), (4, 1, 128, 128, 4), (2, 2, 64, 64, 3), (3, 1, 64, 128, 2), (2, 1, 128, 64, 4),
                              (1, 1, 200, 96, 5), (2, 1, 256, 132, 4), (16, 8, 128, 128, 4)):
        C, rows = 2 * KV * D + H * V, (2 * KV * D + 2 * H * V + 2 * H + 7) // 8 * 8
        p = rnd(T, rows)
        conv, rate, dtb, norm = f32(C, taps) * 0.5, torch.exp(f32(H) - 1.0), f32(H) - 2.0, f32(V)
        state = f32(S + 3, (H * D * V + (taps * C if taps > 1 else 0) + 3) // 4 * 4) * 0.3
        if H == 16:                                               # the many-head case is for speed's sake cut short
            if T > 300:
                continue
        sa = state.clone()
        want = ref.gated_delta_mix(p, conv, taps, rate, dtb, H, KV, D, V, 1e-6, norm, 1e-5, sa, cpu)
        for fused in (True, False):
            ops.fused_delta_step, sb = fused, state.to(dev)
            try:
                got = ops.gated_delta_mix(mv(p), mv(conv), taps, mv(rate), mv(dtb), H, KV, D, V, 1e-6, mv(norm), 1e-5, sb, gpu_b,
                                          chunks=chunk_lists(lens, dev) if fused else None)
            finally:
                ops.fused_delta_step = True
            assert close(got, want) and close(sb, sa, 1e-4 if dtype == torch.float32 else 5e-3), (H, KV, D, V, taps, fused)
    ops.check_errors()


@gpu
@pytest.mark.parametrize("D,V", [(64, 64), (64, 128), (128, 64), (128, 128)])
def test_chunks_against_token_by_token(D, V):
    """The scan in chunks on the tensor cores against the float32 scan of the same rows: entries that end inside a chunk, at its edge and one
    behind it, single tokens among them; decays that forget at once, hardly ever, and per head; keys that repeat (I + A far from the unit
    matrix); states that earlier steps left; scratch that holds one head, two heads or all."""
    ops, dev = cuda_ops(), "cuda:0"
    g = torch.Generator().manual_seed(D + V)
    lens, H, KV = [64, 1, 65, 63, 200, 2, 129], 6, 2
    T, S, C = sum(lens), len(lens), 2 * KV * D + H * V
    starts = [sum(lens[:i]) for i in range(S + 1)]
    batch = SimpleNamespace(num_segs=S, seg_q_start=_i32(starts, dev), seg_slot=_i32([3, 1, 7, 2, 5, 6, 4], dev))
    prep = torch.zeros(T, (C + 3 * H + 3) // 4 * 4)
    unit = torch.nn.functional.normalize
    few = unit(torch.randn(5, D, generator=g), dim=-1)                                     # keys that come again and again
    k = torch.where(torch.rand(T, KV, 1, generator=g) < 0.5, few[torch.randint(0, 5, (T, KV), generator=g)], unit(torch.randn(T, KV, D, generator=g), dim=-1))
    prep[:, :KV * D] = (unit(torch.randn(T, KV, D, generator=g), dim=-1) * D ** -0.5).reshape(T, -1)
    prep[:, KV * D:2 * KV * D] = k.reshape(T, -1)
    prep[:, 2 * KV * D:C] = torch.randn(T, H * V, generator=g)
    prep[:, C:C + H] = torch.rand(T, H, generator=g) * 0.98 + 0.01
    lf = -torch.tensor([1e-6, 1e-3, 0.03, 0.5, 6.0, 60.0]) * (torch.rand(T, H, generator=g) + 0.5)
    prep[:, C + H:C + 2 * H], prep[:, C + 2 * H:C + 3 * H] = lf.exp(), lf
    prep, state = prep.to(dev), torch.randn(9, H * D * V + 8, generator=g).to(dev) * 0.2
    want_state, lists = state.clone(), chunk_lists(lens, dev)
    want = ops.gated_delta_scan(prep, H, KV, D, V, want_state, batch)
    kept = ops.delta_work_bytes
    for heads in (1, 4, 6):
        got_state = state.clone()
        ops.delta_work_bytes = heads * lists[0].shape[0] * int(ops.lib.mi_delta_chunk_bytes(D, V))
        try:
            before = ops.launches
            got = ops.gated_delta_scan(prep, H, KV, D, V, got_state, batch, lists)
            assert ops.launches - before == 2 * -(-H // heads)                             # the chunked form ran
        finally:
            ops.delta_work_bytes = kept
        for h in range(H):
            a, b = got.view(T, H, V)[:, h], want.view(T, H, V)[:, h]
            assert (a - b).abs().max() < 2e-4 * b.abs().max(), (heads, h)
        assert (got_state - want_state).abs().max() < 2e-4 * want_state.abs().max()
        assert torch.equal(got_state[0], state[0]) and torch.equal(got_state[8], state[8])      # slots of nobody
    ops.check_errors()


def plain_judged(d, prompts, got):
    """Generated tokens judged by the plain logits: each is within a rounding's reach of the largest."""
    for p, out in zip(prompts, got):
        logits = JUDGE.logits(d, p + out)
        for i, tok in enumerate(out):
            row = logits[len(p) + i - 1]
            assert row[tok] >= row.max() - 0.2 * row.abs().max()


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
        assert got == [JUDGE.greedy(d, p, 12) for p in prompts]
    else:
        plain_judged(d, prompts, got)


@gpu
def test_long_decoding_on_gpu(dirs):
    """300 tokens generated one by one after a short prompt, through the scheduler: pages fill, the rings of inputs turn many times, and
    the plain implementation agrees on the whole sequence at the end."""
    d, cfg, page = dirs["pages"]
    prompt = tokens(cfg["vocab"], 11, seed=77)
    llm = LLM(d, dtype="float32", kv_block_size=page, kv_cache_tokens=512, max_num_seqs=2)
    out = llm.generate([prompt], SamplingParams(max_new_tokens=300, ignore_eos=True))[0]
    logits = JUDGE.logits(d, prompt + out)
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
        want = JUDGE.logits(d, a)
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
    assert data["summary"]["engine"]["architecture"] == "Kofutar"
    assert all(run["generated_tokens"] == 9 and run["error"] is None for run in data["runs"])

"""Fetodra: configuration -> ModelSpec.

A decoder with the norms behind the sums, x <- N(alpha x + sublayer(x)) (1 + w), whose layers are chosen one by one from two
mixers: grouped softmax attention whose projections pass a short causal convolution (queries and keys then normed over the
whole projection and partly rotated; scores capped; a window with the first tokens kept; the heads' outputs gated), and Mamba-2
(a state-space recurrence with one decay per head).  An attention layer may read the keys and values of an earlier one instead
of making its own.  The feed-forward is a clamped gated one, or none.  The stream is float32.
Tensor names are the checkpoint's own: embed, l<i>.norm1, l<i>.mix.*, l<i>.norm2, l<i>.mlp.*, final.norm, head.
"""
from __future__ import annotations

from ..config.fetodra_config import FetodraConfig
from ..config.registry import register_architecture
from ..config.spec import ExecStep, LayerSpec, ModelSpec, PartSpec

GATE_SLOPE = 1.702                  # the feed-forward's gate is g * sigmoid(GATE_SLOPE g)


def _mixer(cfg: FetodraConfig, kind: str, m: dict):
    """(PartSpec of the mixer, PartSpec of its position encoding, its tensors)."""
    if kind == "mamba2":
        spec = PartSpec.of("mamba2", hidden_size=cfg.width, num_heads=m["heads"], value_dim=m["vdim"], state_dim=m["state"], groups=m["groups"],
                           norm_groups=m["norm_groups"], conv_taps=m["conv"], out_norm_eps=cfg.norm_eps)
        return spec, PartSpec.of("none"), ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")
    borrows = "kv_from" in m
    mask = m.get("mask") or {}
    spec = PartSpec.of("filtered_attention", hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"],
                       value_dim=m["vdim"], scale=m["scale"], conv_taps=m["conv"], norm_eps=cfg.norm_eps, softcap=m.get("softcap"),
                       window=mask.get("size"), keep_first=mask.get("keep_first", 0), borrows_keys=borrows)
    tensors = [n + s for n in (("q",) if borrows else ("q", "k", "v")) for s in ("", ".b", ".conv")]
    tensors += ["q.norm"] if borrows else ["q.norm", "k.norm"]
    return spec, PartSpec.of("rotary_interleaved", dims=m["rot"]["dims"], theta=m["rot"]["base"]), tuple(tensors) + ("g", "o")


def build_spec(cfg: FetodraConfig) -> ModelSpec:
    norm = PartSpec.of("sum_rmsnorm", size=cfg.width, eps=cfg.norm_eps, alpha=cfg.postln_alpha, one_plus=True)
    layers, order = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer_dict()
        mixer, position, tensors = _mixer(cfg, layer.type, m)
        names = {"norm1.weight": p + "norm1"}
        names.update({f"mixer.{t}": p + "mix." + t for t in tensors})
        parts = dict(mixer=mixer, norm1=norm, position=position)
        block = "postnorm_mixer"
        if layer.mlp is not None:
            block = "postnorm"
            parts.update(norm2=norm, feed_forward=PartSpec.of("clamped_mlp", hidden_size=cfg.width, intermediate_size=layer.mlp.ff,
                                                              limit=layer.mlp.limit, gate_slope=GATE_SLOPE))
            names["norm2.weight"] = p + "norm2"
            names.update({f"feed_forward.{t}": p + "mlp." + t for t in ("gate", "up", "down")})
        layers.append(LayerSpec.of(block, names, **parts))
        order.append(ExecStep(i, cache_from=m.get("kv_from")))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, layers=tuple(layers), order=tuple(order),
        final_norm=PartSpec.of("stream_rmsnorm", size=cfg.width, eps=cfg.norm_eps, one_plus=True), embedding_name="embed",
        final_norm_name="final.norm", lm_head_name="head", max_position=cfg.max_position, residual="float32")


register_architecture("Fetodra", "Fetodra (convolution-filtered attention with a score cap and shared keys / Mamba-2 layers, norms behind the sums, "
                      "clamped feed-forward, float32 stream)", FetodraConfig, build_spec)

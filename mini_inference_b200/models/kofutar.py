"""Kofutar: configuration -> ModelSpec.

A decoder whose layers are chosen one by one from three mixers (a delta rule with one decay per head; grouped softmax attention with
normed, partly rotated queries and keys; latent attention with a query latent, a learned sink and an output gate), each followed by a
dense feed-forward with a gelu gate, or by none.  Every sublayer stands between two layer norms: the stream is normed on its way in and the
output on its way out, before it is added.  A span of layers may run several times with the same weights, each pass with caches and
states of its own and behind a product that reads the stream beside the embedded tokens.  The stream is float32.
Tensor names are the checkpoint's own: embed, loop.in, l<i>.norm1, l<i>.norm1b, l<i>.mix.*, l<i>.norm2, l<i>.norm2b, l<i>.mlp.*,
final.norm, head.
"""
from __future__ import annotations

from ..config.kofutar_config import KofutarConfig
from ..config.registry import register_architecture
from ..config.spec import ExecStep, LayerSpec, ModelSpec, PartSpec

# constants the design fixes
UNIT_EPS = 1e-6                     # added to the sum of squares inside the root of the delta rule's unit vectors

_MIXER_TENSORS = {
    "delta": ("q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "A_log", "norm", "a", "dt_bias", "g", "o"),
    "attention": ("q", "k", "v", "q.norm", "k.norm", "o"),
    "latent_attention": ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "sink", "g", "o"),
}


def execution_order(num_layers: int, loop):
    """Layers before the repeated span once, the span `times` times (the first layer of every pass is marked: the stream is joined
    with the embedded tokens before it), the rest once."""
    if loop is None:
        return tuple(ExecStep(i) for i in range(num_layers))
    start, stop, times = loop
    order = [ExecStep(i) for i in range(start)]
    for _ in range(times):
        order += [ExecStep(i, join_embedding=i == start) for i in range(start, stop)]
    return tuple(order + [ExecStep(i) for i in range(stop, num_layers)])


def _position(rot: dict) -> PartSpec:
    return PartSpec.of("rotary_half", dims=rot["dims"], theta=rot["base"], factor=(rot.get("scaling") or {}).get("factor", 1.0))


def _mixer(cfg: KofutarConfig, kind: str, m: dict):
    """(PartSpec of the mixer, of its positions)."""
    if kind == "delta":
        return PartSpec.of("gated_delta", hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"],
                           value_dim=m["vdim"], conv_taps=m["conv"], out_norm_eps=cfg.norm_eps, unit_eps=UNIT_EPS), PartSpec.of("none")
    if kind == "attention":
        return PartSpec.of("sink_attention", hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"],
                           value_dim=m["vdim"], scale=m["scale"], unit_norm_eps=cfg.norm_eps, norm_weights=True, rotate=True), _position(m["rot"])
    return PartSpec.of("latent_attention", hidden_size=cfg.width, num_heads=m["heads"], nope_dim=m["dim"], rot_dim=m["rot_dim"],
                       value_dim=m["vdim"], kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=m["scale"], latent_norm_eps=cfg.norm_eps,
                       gate="elements", sink=True), _position(m["rot"])


def build_spec(cfg: KofutarConfig) -> ModelSpec:
    norm = PartSpec.of("stream_layernorm", size=cfg.width, eps=cfg.norm_eps)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        mixer, position = _mixer(cfg, layer.type, layer.mixer_dict())
        names = {"norm1.weight": p + "norm1", "norm1b.weight": p + "norm1b"}
        names.update({f"mixer.{t}": p + "mix." + t for t in _MIXER_TENSORS[layer.type]})
        parts = dict(mixer=mixer, norm1=norm, norm1b=norm, position=position)
        block = "sandwich_mixer"
        if layer.ff is not None:
            block = "sandwich"
            parts.update(norm2=norm, norm2b=norm,
                         feed_forward=PartSpec.of("gated_mlp", hidden_size=cfg.width, intermediate_size=layer.ff, act="gelu_tanh"))
            names.update({"norm2.weight": p + "norm2", "norm2b.weight": p + "norm2b"})
            names.update({f"feed_forward.{t}": p + "mlp." + t for t in ("gate", "up", "down")})
        layers.append(LayerSpec.of(block, names, **parts))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, layers=tuple(layers), order=execution_order(len(layers), cfg.loop), final_norm=norm,
        embedding_name="embed", final_norm_name="final.norm", lm_head_name="head", max_position=cfg.max_position, residual="float32",
        join_name="loop.in" if cfg.loop is not None else None)


register_architecture("Kofutar", "Kofutar (delta-rule / rotated attention / latent attention layers between two layer norms, looped span that "
                      "reads the embedded tokens again, float32 stream)", KofutarConfig, build_spec)

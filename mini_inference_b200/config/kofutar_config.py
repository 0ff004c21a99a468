"""Typed configuration of the Kofutar design, read from its own config.json keys.

config.json names every size and every constant that differs between models of the design:
  architecture        "Kofutar"
  vocab, width        vocabulary and width of the residual stream
  norm.eps            the one epsilon of all layer norms and root-mean-square norms
  loop                {start, stop, times}: layers start .. stop-1 run `times` times in a row, each pass behind a product that joins
                      the stream with the embedded tokens (absent or null: every layer once, no such product)
  layers[i]           type ("delta" | "attention" | "latent_attention"), mixer {sizes and constants of that mixer}, and
                      mlp: null (no feed-forward) or {"kind": "dense", "ff": n}
    delta               heads, kv_heads, dim, vdim, conv
    attention           heads, kv_heads, dim, vdim, scale, rot {base, dims, scaling {factor} (optional)}
    latent_attention    heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot {base, dims, scaling {factor} (optional)}
A missing key is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .json_keys import frozen, need, positive, thawed
from .model_config import ConfigError

MIXER_KEYS = {
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "rot"),
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot"),
}


@dataclass(frozen=True)
class KofutarLayer:
    type: str
    mixer: tuple                                  # nested objects as sorted (key, value) pairs
    ff: Optional[int]                             # intermediate size of the dense feed-forward (None: the layer has none)

    def mixer_dict(self) -> dict:
        return thawed(self.mixer)


def _read_rotation(mx: dict, rotatable: int, where: str) -> dict:
    rot = dict(mx["rot"])
    need(rot, ("base", "dims"), where)
    if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= rotatable:
        raise ConfigError(f"config.json: {where}.dims must be an even number up to {rotatable}")
    if rot.get("scaling") is not None:
        need(rot["scaling"], ("factor",), f"{where}.scaling")
        if not float(rot["scaling"]["factor"]) > 0:
            raise ConfigError(f"config.json: {where}.scaling.factor must be positive")
    else:
        rot.pop("scaling", None)
    return rot


def _read_mixer(kind: str, mx: dict, where: str) -> dict:
    need(mx, MIXER_KEYS[kind], where)
    positive(mx, [k for k in MIXER_KEYS[kind] if k not in ("scale", "rot", "rot_dim")], where)
    if "kv_heads" in MIXER_KEYS[kind] and int(mx["heads"]) % int(mx["kv_heads"]):
        raise ConfigError(f"config.json: {where}: {mx['heads']} heads are not a multiple of {mx['kv_heads']} kv_heads")
    if kind != "delta":
        mx = dict(mx, rot=_read_rotation(mx, int(mx["rot_dim" if kind == "latent_attention" else "dim"]), f"{where}.rot"))
    return mx


def _read_ff(mlp, where: str) -> Optional[int]:
    if mlp is None:
        return None
    need(mlp, ("kind",), where)
    if mlp["kind"] != "dense":
        raise ConfigError(f"config.json: {where}.kind '{mlp['kind']}' is not dense")
    need(mlp, ("ff",), where)
    positive(mlp, ("ff",), where)
    return int(mlp["ff"])


@dataclass(frozen=True)
class KofutarConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    loop: Optional[Tuple[int, int, int]]          # start, stop, times
    layers: Tuple[KofutarLayer, ...]
    max_position: int = 1 << 20                   # the design tabulates no positions: an engine limit only

    @classmethod
    def from_dict(cls, raw: dict) -> "KofutarConfig":
        need(raw, ("vocab", "width", "layers", "norm"), "the top level")
        need(raw["norm"], ("eps",), "'norm'")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            need(entry, ("type", "mixer"), where)
            kind = entry["type"]
            if kind not in MIXER_KEYS:
                raise ConfigError(f"config.json: {where} has type '{kind}' (known: {', '.join(sorted(MIXER_KEYS))})")
            layers.append(KofutarLayer(kind, frozen(_read_mixer(kind, dict(entry["mixer"]), f"{where}.mixer")),
                                       _read_ff(entry.get("mlp"), f"{where}.mlp")))
        loop = raw.get("loop")
        if loop is not None:
            need(loop, ("start", "stop", "times"), "'loop'")
            loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if not (0 <= loop[0] < loop[1] <= len(layers)) or loop[2] < 1:
                raise ConfigError(f"config.json: loop {loop} does not fit {len(layers)} layers")
        return cls(architecture=raw.get("architecture") or (raw.get("architectures") or ["Kofutar"])[0],
                   vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]), loop=loop, layers=tuple(layers),
                   max_position=int(raw.get("max_position", 1 << 20)))

    def to_dict(self) -> dict:
        layers = [{"type": layer.type, "mixer": layer.mixer_dict(), "mlp": None if layer.ff is None else {"kind": "dense", "ff": layer.ff}}
                  for layer in self.layers]
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "layers": layers}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return out

    def describe(self) -> dict:
        return {"architecture": self.architecture, "loop": self.loop,
                "layers": [f"{layer.type}+{'dense' if layer.ff else 'none'}" for layer in self.layers]}

"""Typed configuration of the Fetodra design, read from its own config.json keys.

config.json names every size and every constant that differs between models of the design:
  architecture        "Fetodra"
  vocab, width        vocabulary and width of the residual stream
  norm.eps            the one epsilon of all root-mean-square norms
  postln_alpha        the stream's weight where a sublayer's output is added to it (the sum is then normed)
  layers[i]           type ("attention" | "mamba2"), mixer {sizes and constants of that mixer}, and
                      mlp: null (no feed-forward) or {"kind": "dense", "ff": n, "limit": c}
    attention         heads, kv_heads, dim, vdim, conv (taps), scale, softcap (absent or null: none), rot {base, dims},
                      mask {size, keep_first} (absent or null: every key), kv_from (absent or null: keys and values of its own;
                      j: those of layer j, an earlier attention layer with keys and values of its own and the same head sizes)
    mamba2            heads, vdim, state, groups, norm_groups, conv (taps)
A missing key is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .json_keys import frozen, need, positive, thawed
from .model_config import ConfigError

MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim", "conv", "scale", "rot"),
    "mamba2": ("heads", "vdim", "state", "groups", "norm_groups", "conv"),
}
SHARED_SIZES = ("heads", "kv_heads", "dim", "vdim", "rot")      # what a layer must have in common with the one whose keys it reads


@dataclass(frozen=True)
class FetodraMLP:
    ff: int
    limit: float


@dataclass(frozen=True)
class FetodraLayer:
    type: str
    mixer: tuple                                  # nested objects as sorted (key, value) pairs
    mlp: Optional[FetodraMLP]

    def mixer_dict(self) -> dict:
        return thawed(self.mixer)


def _read_attention(mx: dict, where: str, index: int, before) -> dict:
    positive(mx, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
    if int(mx["heads"]) % int(mx["kv_heads"]):
        raise ConfigError(f"config.json: {where}: {mx['heads']} heads are not a multiple of {mx['kv_heads']} kv_heads")
    need(mx["rot"], ("base", "dims"), f"{where}.rot")
    if int(mx["rot"]["dims"]) % 2 or not 0 <= int(mx["rot"]["dims"]) <= int(mx["dim"]):
        raise ConfigError(f"config.json: {where}.rot.dims must be an even number up to dim")
    if mx.get("mask") is not None:
        need(mx["mask"], ("size",), f"{where}.mask")
        mask = {"size": int(mx["mask"]["size"]), "keep_first": int(mx["mask"].get("keep_first") or 0)}
        if mask["size"] < 1 or mask["keep_first"] < 0:
            raise ConfigError(f"config.json: {where}.mask: a window of {mask['size']} keys with the first {mask['keep_first']} kept")
        mx["mask"] = mask
    for k in ("mask", "softcap", "kv_from"):
        if mx.get(k) is None:
            mx.pop(k, None)
    if "softcap" in mx and not float(mx["softcap"]) > 0:
        raise ConfigError(f"config.json: {where}.softcap must be positive")
    if "kv_from" in mx:
        j = int(mx["kv_from"])
        if not 0 <= j < index or before[j].type != "attention" or "kv_from" in before[j].mixer_dict():
            raise ConfigError(f"config.json: {where}.kv_from is {j}: not an earlier attention layer with keys and values of its own")
        other = before[j].mixer_dict()
        differ = [k for k in SHARED_SIZES if other[k] != mx[k]]
        if differ:
            raise ConfigError(f"config.json: {where} reads the keys of layer {j}, which differs in {', '.join(differ)}")
    return mx


def _read_mamba2(mx: dict, where: str) -> dict:
    positive(mx, MIXER_KEYS["mamba2"], where)
    if int(mx["heads"]) % int(mx["groups"]):
        raise ConfigError(f"config.json: {where}: {mx['heads']} heads are not a multiple of {mx['groups']} groups")
    if int(mx["heads"]) * int(mx["vdim"]) % int(mx["norm_groups"]):
        raise ConfigError(f"config.json: {where}: {mx['heads']} heads of {mx['vdim']} do not part into norm_groups = {mx['norm_groups']}")
    return mx


@dataclass(frozen=True)
class FetodraConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    postln_alpha: float
    layers: Tuple[FetodraLayer, ...]
    max_position: int = 1 << 20                   # the design tabulates no positions: an engine limit only

    @classmethod
    def from_dict(cls, raw: dict) -> "FetodraConfig":
        need(raw, ("vocab", "width", "layers", "norm", "postln_alpha"), "the top level")
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
            mx = dict(entry["mixer"])
            need(mx, MIXER_KEYS[kind], f"{where}.mixer")
            mx = _read_attention(mx, f"{where}.mixer", i, layers) if kind == "attention" else _read_mamba2(mx, f"{where}.mixer")
            mlp = entry.get("mlp")
            if mlp is not None:
                need(mlp, ("kind", "ff", "limit"), f"{where}.mlp")
                if mlp["kind"] != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind '{mlp['kind']}' is not dense")
                mlp = FetodraMLP(int(mlp["ff"]), float(mlp["limit"]))
            layers.append(FetodraLayer(kind, frozen(mx), mlp))
        return cls(architecture=raw.get("architecture") or (raw.get("architectures") or ["Fetodra"])[0],
                   vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]),
                   postln_alpha=float(raw["postln_alpha"]), layers=tuple(layers), max_position=int(raw.get("max_position", 1 << 20)))

    def to_dict(self) -> dict:
        layers = [{"type": layer.type, "mixer": layer.mixer_dict(),
                   "mlp": None if layer.mlp is None else {"kind": "dense", "ff": layer.mlp.ff, "limit": layer.mlp.limit}} for layer in self.layers]
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "postln_alpha": self.postln_alpha, "layers": layers}

    def describe(self) -> dict:
        def kind(layer):
            shared = layer.mixer_dict().get("kv_from")
            return layer.type + ("" if shared is None else f"(keys of {shared})") + ("+dense" if layer.mlp else "+none")
        return {"architecture": self.architecture, "layers": [kind(layer) for layer in self.layers]}

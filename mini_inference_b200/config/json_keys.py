"""Reading config.json objects: required keys with an error that names what is missing, and nested objects as hashable values."""
from __future__ import annotations

from .model_config import ConfigError


def need(d, keys, where: str):
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    missing = [k for k in keys if d.get(k) is None]
    if missing:
        raise ConfigError(f"config.json: {where} lacks {', '.join(missing)}")


def positive(d: dict, keys, where: str):
    for k in keys:
        if int(d[k]) < 1:
            raise ConfigError(f"config.json: {where}.{k} must be at least 1")


def frozen(value):
    """Nested objects as sorted (key, value) pairs, lists as tuples."""
    if isinstance(value, dict):
        return tuple(sorted((k, frozen(v)) for k, v in value.items()))
    if isinstance(value, list):
        return tuple(frozen(v) for v in value)
    return value


def thawed(value):
    """The objects behind `frozen`."""
    if isinstance(value, tuple) and all(isinstance(v, tuple) and len(v) == 2 and isinstance(v[0], str) for v in value):
        return {k: thawed(v) for k, v in value}
    return value

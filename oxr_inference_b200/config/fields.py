"""Reading single values out of a config.json, with errors that name the place."""

from __future__ import annotations

from typing import Any, Mapping

from oxr_inference_b200.config.model_config import ConfigError


def need(d: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(d, Mapping) or key not in d:
        raise ConfigError(f"config.json: {where} lacks {key!r}")
    return d[key]


def pos_int(d: Mapping[str, Any], key: str, where: str) -> int:
    v = need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"config.json: {where}.{key} must be a positive integer, got {v!r}")
    return v


def nonneg_int(d: Mapping[str, Any], key: str, where: str) -> int:
    v = need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"config.json: {where}.{key} must be an integer >= 0, got {v!r}")
    return v


def number(d: Mapping[str, Any], key: str, where: str) -> float:
    v = need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
    return float(v)

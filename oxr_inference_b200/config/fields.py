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


def head_counts(d: Mapping[str, Any], where: str) -> dict[str, int]:
    """``heads`` and ``kv_heads`` of a grouped-query mixer entry, which must divide."""
    out = {"num_heads": pos_int(d, "heads", where), "num_kv_heads": pos_int(d, "kv_heads", where)}
    if out["num_heads"] % out["num_kv_heads"]:
        raise ConfigError(f"config.json: {where}: {out['num_heads']} heads are not a multiple of {out['num_kv_heads']} kv_heads")
    return out


def weights_owner(listed: list, i: int) -> int:
    """Follow ``weights_of`` from layer i of a config.json's ``layers`` to the layer that has tensors."""
    seen = {i}
    at = i
    while isinstance(listed[at], Mapping) and listed[at].get("weights_of") is not None:
        j = listed[at]["weights_of"]
        if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < len(listed) or j in seen:
            raise ConfigError(f"config.json: layers[{at}].weights_of must name another layer that has tensors, got {j!r}")
        seen.add(j)
        at = j
    return at


def number(d: Mapping[str, Any], key: str, where: str) -> float:
    v = need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
    return float(v)

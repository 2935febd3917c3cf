"""Finolix: a decoder of several residual streams whose config.json lists its layers one by one, from typed config to a description made of
registered parts.

Every sublayer reads the RMS norm (weight stored around zero) of a weighted sum of the streams; its result, scaled entry by entry, goes to every
stream with that stream's weight while a small matrix mixes the streams (hyper-connections). All streams start as the embedding's output, and
their sum is what the final norm and the untied head read. Two mixers. ``latent_attention``: attention over one cached row per token, a normed
latent beside a rotated key part that all heads share, within a sliding window and with a sink per head; the queries pass a normed latent of their
own; neighbouring entries of the rotated part form a pair, and a YaRN ramp rescales the frequencies. ``attention``: causal grouped-query
attention with weighted q/k norm, a rotation of the first ``rot.dims`` entries in the half-split layout, and one sigmoid gate per head.
Feed-forwards: none, a two-matrix layer with the square of relu (``dense``), or routed SiLU-gated experts (``moe``) picked by biased logits
and weighted by the softmax over the chosen ones. A layer with ``weights_of: j`` runs layer j's tensors with a cache of its own.

Tensor names: ``embed``, ``head``, ``final.norm``, and per layer ``l<i>.{norm1,norm2,ls1,ls2}``, ``l<i>.hc1.{in,out,mix}``, ``l<i>.hc2.{in,out,mix}``,
``l<i>.mix.*`` and ``l<i>.mlp.*``: ``mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,o}``; ``mix.{q,k,v,q.norm,k.norm,g,o}``; ``mlp.{up,down}`` or
``mlp.{router,router.b,e<j>.{gate,up,down}}``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from oxr_inference_b200.config.fields import head_counts, need, nonneg_int, number, pos_int, weights_owner
from oxr_inference_b200.config.model_config import ConfigError
from oxr_inference_b200.config.registry import Architecture, register_architecture
from oxr_inference_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 20
"""The design has no table over positions and config.json gives no limit; this bounds a request's length for the scheduler."""
MAX_STREAMS = 16
"""What the kernels that mix the streams are built for."""


@dataclass(frozen=True)
class FinolixLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None
    owner: int
    """The layer whose tensors this one runs with (itself, unless the entry has ``weights_of``)."""


@dataclass(frozen=True)
class FinolixConfig:
    width: int
    vocab: int
    eps: float
    streams: int
    layers: tuple[FinolixLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = "Finolix"

    @staticmethod
    def from_dict(raw: Mapping[str, Any], generation: Mapping[str, Any] | None = None) -> "FinolixConfig":
        listed = need(raw, "layers", "the top level")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = need(entry, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not one of {sorted(_MIXERS)}")
            mlp = entry.get("mlp")
            if mlp is not None and need(mlp, "kind", where + ".mlp") not in _FEED_FORWARDS:
                raise ConfigError(f"config.json: {where}.mlp.kind {mlp['kind']!r} is not one of {sorted(_FEED_FORWARDS)}")
            layers.append(FinolixLayer(kind, dict(need(entry, "mixer", where)), dict(mlp) if mlp is not None else None, weights_owner(listed, i)))
        for i, layer in enumerate(layers):
            theirs = layers[layer.owner]
            if (layer.type, layer.mixer, layer.mlp) != (theirs.type, theirs.mixer, theirs.mlp):
                raise ConfigError(f"config.json: layers[{i}] runs with layer {layer.owner}'s tensors but does not describe the same layer")
        streams = pos_int(raw, "streams", "the top level")
        if streams > MAX_STREAMS:
            raise ConfigError(f"config.json: {streams} streams; up to {MAX_STREAMS} are implemented")
        eos = raw.get("eos_token_id", [])
        if generation is not None and generation.get("eos_token_id") is not None:
            eos = generation["eos_token_id"]
        eos = [] if eos is None else (list(eos) if isinstance(eos, list) else [eos])
        config = FinolixConfig(
            width=pos_int(raw, "width", "the top level"), vocab=pos_int(raw, "vocab", "the top level"),
            eps=number(need(raw, "norm", "the top level"), "eps", "norm"), streams=streams, layers=tuple(layers),
            eos_token_ids=tuple(int(t) for t in eos), architecture=str(raw.get("architecture", "Finolix")))
        finolix_model_spec(config)   # sizes that do not fit each other are config errors, found here
        return config


# ---- the pieces of a mixer entry
def _rotation(kind: str, m: Mapping[str, Any], where: str, entries: int) -> PartSpec | None:
    """The ``rot`` entry of a mixer as a rotation within ``entries`` entries in the layout ``kind``, None without one."""
    rot = m.get("rot")
    if not rot:
        return None
    where += ".rot"
    dims, base = pos_int(rot, "dims", where), number(rot, "base", where)
    if dims % 2 or dims > entries:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {entries}")
    if not base > 1:
        raise ConfigError(f"config.json: {where}.base must be above 1")
    params: dict[str, Any] = {"dims": dims, "base": base}
    scaling = rot.get("scaling")
    if scaling:
        values = {name: number(scaling, name, where + ".scaling") for name in ("factor", "original", "fast", "slow")}
        if not all(v > 0 for v in values.values()):
            raise ConfigError(f"config.json: {where}.scaling: every value must be positive")
        params["scaling"] = {"kind": "ramp", **values}
    return PartSpec(kind, params)


# ---- one function per mixer kind: (config, layer index) -> (mixer part, position part or None)
def _latent(c: FinolixConfig, i: int) -> tuple[PartSpec, PartSpec | None]:
    m, where = c.layers[i].mixer, f"layers[{i}].mixer"
    rot_dim = nonneg_int(m, "rot_dim", where)
    position = _rotation("rope_pairs", m, where, rot_dim) if rot_dim else None
    if rot_dim and (position is None or position.params["dims"] != rot_dim):
        raise ConfigError(f"config.json: {where}.rot.dims must be the {rot_dim} entries of the rotated part")
    return PartSpec("latent_attention", {
        "hidden_size": c.width, "num_heads": pos_int(m, "heads", where), "key_dim": pos_int(m, "dim", where), "rot_dim": rot_dim,
        "value_dim": pos_int(m, "vdim", where), "rank": pos_int(m, "kv_rank", where), "q_rank": pos_int(m, "q_rank", where),
        "scale": number(m, "scale", where), "eps": c.eps, "sink": True,
        "window": pos_int(m["mask"], "size", where + ".mask") if m.get("mask") else 0}, prefix=f"l{i}.mix."), position


def _gated(c: FinolixConfig, i: int) -> tuple[PartSpec, PartSpec | None]:
    m, where = c.layers[i].mixer, f"layers[{i}].mixer"
    dim = pos_int(m, "dim", where)
    return PartSpec("gated_attention", {
        "hidden_size": c.width, **head_counts(m, where), "key_dim": dim, "value_dim": pos_int(m, "vdim", where), "scale": number(m, "scale", where),
        "eps": c.eps, "qk_norm": "weighted", "output_gate": "head"}, prefix=f"l{i}.mix."), _rotation("rope_halves", m, where, dim)


_MIXERS = {"latent_attention": _latent, "attention": _gated}


# ---- one function per feed-forward kind
def _dense(c: FinolixConfig, mlp: Mapping[str, Any], prefix: str) -> PartSpec:
    return PartSpec("relu2_mlp", {"hidden_size": c.width, "intermediate_size": pos_int(mlp, "ff", prefix + "mlp")}, prefix=prefix + "mlp.")


def _experts(c: FinolixConfig, mlp: Mapping[str, Any], prefix: str) -> PartSpec:
    where = prefix + "mlp"
    router = need(mlp, "router", where)
    params = {"hidden_size": c.width, "intermediate_size": pos_int(need(mlp, "expert", where), "ff", where + ".expert"),
              "experts": pos_int(router, "experts", where + ".router"), "top": pos_int(router, "top", where + ".router"), "activation": "silu_glu",
              "score": "chosen_softmax", "router_bias": True}
    if params["top"] > params["experts"]:
        raise ConfigError(f"config.json: {where}.router: {params['top']} of {params['experts']} experts cannot be chosen")
    return PartSpec("routed_experts", params, prefix=prefix + "mlp.")


_FEED_FORWARDS = {"dense": _dense, "moe": _experts}


def finolix_model_spec(c: FinolixConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec("rms_norm", {"size": c.width, "eps": c.eps, "around_zero": True}, prefix=name, names={"weight": ""})

    layers: list[LayerSpec] = []
    index: dict[int, int] = {}     # layer with tensors -> its place among the spec's layers
    for i, layer in enumerate(c.layers):
        if layer.owner != i:
            continue
        p = f"l{i}."
        mixer, position = _MIXERS[layer.type](c, i)
        ff = _FEED_FORWARDS[layer.mlp["kind"]](c, layer.mlp, p) if layer.mlp is not None else None
        index[i] = len(layers)
        layers.append(LayerSpec(
            mixer=mixer, mixer_norm=norm(p + "norm1"), feed_forward=ff, feed_forward_norm=norm(p + "norm2") if ff else None, position=position,
            block=PartSpec("hyper_connections", {"hidden_size": c.width, "streams": c.streams, "layer_scale": True}, prefix=p)))
    return ModelSpec(
        architecture=c.architecture, hidden_size=c.width, vocab_size=c.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": c.width, "scale": 1.0, "whole_stream": True},
                           prefix="embed", names={"weight": ""}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(index[layer.owner]) for layer in c.layers),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": c.vocab, "hidden_size": c.width, "tied": False}, prefix="head", names={"weight": ""}),
        max_positions=MAX_POSITIONS, eos_token_ids=c.eos_token_ids,
        # a layer without a feed-forward may still carry the norm, the scale and the stream weights of one
        ignored_tensors=(r"l\d+\.(norm2|ls2|hc2\.(in|out|mix))",))


FINOLIX = register_architecture(Architecture("Finolix", FinolixConfig.from_dict, finolix_model_spec))

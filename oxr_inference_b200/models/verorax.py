"""Verorax: a decoder whose config.json lists its layers one by one, from typed config to a description made of registered parts.

Every layer is ``x += norm1b(mixer(g))`` and, unless its ``mlp`` is null, ``x += norm2b(ff(norm2(x)))``, where g is ``h = norm1(x)`` moved the share ``shift`` of
the way to the previous token's h, entry by entry (RMS norms with weights; the previous h belongs to a sequence's state). Three mixers.
``latent_attention``: causal attention over one cached row per token, a normed latent beside a rotated key part that all heads share; the
queries pass a normed latent of their own. ``attention``: differential attention with biases and a window, no rotation. ``parallel``: two mixers
side by side, ``left_scale * left + right_scale * right``: windowed grouped-query attention with weighted q/k norm, a rotation of the first ``rot.dims``
entries in the half-split layout, a learned temperature and a sigmoid gate per head; and a generalized delta rule with a decay per key
channel. Feed-forwards: a GELU-gated layer (``dense``) or routed SiLU-gated experts (``moe``) chosen by the softmax score plus a learned
correction, weighted by the score alone, with ``router.identity`` more experts behind them that return their input. A layer with ``weights_of: j`` runs
layer j's tensors with a cache and state of its own. The model ends in an RMS norm and an untied head.

Tensor names: ``embed``, ``head``, ``final.norm``, and per layer ``l<i>.{norm1,norm1b,norm2,norm2b,shift}``, ``l<i>.mix.*`` and ``l<i>.mlp.*``:
``mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}``; ``mix.{q,k,v}``, ``mix.{q,k,v}.b``, ``mix.{lq1,lk1,lq2,lk2,o}``; ``mix.left.{q,k,v,q.norm,k.norm,temp,g,o}`` and
``mix.right.{r,k,v,g,a,a.b,w1,w2,w0,norm,o}``; ``mlp.{gate,up,down}`` or ``mlp.{router,correction,e<j>.{gate,up,down}}``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from oxr_inference_b200.config.fields import head_counts, need, nonneg_int, number, pos_int, weights_owner
from oxr_inference_b200.config.model_config import ConfigError
from oxr_inference_b200.config.registry import Architecture, register_architecture
from oxr_inference_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

DECAY_RANK = 16
"""Width of the decay's low-rank map where nothing says it: config.json does not give it, a checkpoint's ``mix.right.w1`` does by its shape
(random-weights mode may name it as ``rank`` in the mixer's ``right`` entry)."""
MAX_POSITIONS = 1 << 20
"""The design has no table over positions and config.json gives no limit; this bounds a request's length for the scheduler."""


@dataclass(frozen=True)
class VeroraxLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None
    owner: int
    """The layer whose tensors this one runs with (itself, unless the entry has ``weights_of``)."""


@dataclass(frozen=True)
class VeroraxConfig:
    width: int
    vocab: int
    eps: float
    layers: tuple[VeroraxLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = "Verorax"

    @staticmethod
    def from_dict(raw: Mapping[str, Any], generation: Mapping[str, Any] | None = None) -> "VeroraxConfig":
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
            layers.append(VeroraxLayer(kind, dict(need(entry, "mixer", where)), dict(mlp) if mlp is not None else None, weights_owner(listed, i)))
        for i, layer in enumerate(layers):
            theirs = layers[layer.owner]
            if (layer.type, layer.mixer, layer.mlp) != (theirs.type, theirs.mixer, theirs.mlp):
                raise ConfigError(f"config.json: layers[{i}] runs with layer {layer.owner}'s tensors but does not describe the same layer")
        eos = raw.get("eos_token_id", [])
        if generation is not None and generation.get("eos_token_id") is not None:
            eos = generation["eos_token_id"]
        eos = [] if eos is None else (list(eos) if isinstance(eos, list) else [eos])
        config = VeroraxConfig(
            width=pos_int(raw, "width", "the top level"), vocab=pos_int(raw, "vocab", "the top level"),
            eps=number(need(raw, "norm", "the top level"), "eps", "norm"), layers=tuple(layers), eos_token_ids=tuple(int(t) for t in eos),
            architecture=str(raw.get("architecture", "Verorax")))
        verorax_model_spec(config)   # sizes that do not fit each other are config errors, found here
        return config


# ---- the pieces of a mixer entry
def _rotation(m: Mapping[str, Any], where: str, entries: int) -> PartSpec | None:
    """The ``rot`` entry of a mixer as a half-split rotation within ``entries`` entries, None without one."""
    rot = m.get("rot")
    if not rot:
        return None
    where += ".rot"
    dims, base = pos_int(rot, "dims", where), number(rot, "base", where)
    if dims % 2 or dims > entries:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {entries}")
    if not base > 1:
        raise ConfigError(f"config.json: {where}.base must be above 1")
    return PartSpec("rope_halves", {"dims": dims, "base": base})


def _window(m: Mapping[str, Any], where: str) -> int:
    return pos_int(m["mask"], "size", where + ".mask") if m.get("mask") else 0


# ---- one function per mixer kind: (config, layer index, checkpoint shapes or None) -> (mixer part, position part or None)
def _latent(c: VeroraxConfig, i: int, shapes) -> tuple[PartSpec, PartSpec | None]:
    m, where, prefix = c.layers[i].mixer, f"layers[{i}].mixer", f"l{i}.mix."
    rot_dim = nonneg_int(m, "rot_dim", where)
    position = _rotation(m, where, rot_dim) if rot_dim else None
    if rot_dim and (position is None or position.params["dims"] != rot_dim):
        raise ConfigError(f"config.json: {where}.rot.dims must be the {rot_dim} entries of the rotated part")
    return PartSpec("latent_attention", {
        "hidden_size": c.width, "num_heads": pos_int(m, "heads", where), "key_dim": pos_int(m, "dim", where), "rot_dim": rot_dim,
        "value_dim": pos_int(m, "vdim", where), "rank": pos_int(m, "kv_rank", where), "q_rank": pos_int(m, "q_rank", where),
        "scale": number(m, "scale", where), "eps": c.eps, "sink": False}, prefix=prefix), position


def _differential(c: VeroraxConfig, i: int, shapes) -> tuple[PartSpec, PartSpec | None]:
    m, where, prefix = c.layers[i].mixer, f"layers[{i}].mixer", f"l{i}.mix."
    return PartSpec("differential_attention", {
        "hidden_size": c.width, **head_counts(m, where), "dim": pos_int(m, "dim", where), "value_dim": pos_int(m, "vdim", where),
        "scale": number(m, "scale", where), "diff": number(m, "diff", where), "eps": c.eps, "window": _window(m, where), "biases": True},
        prefix=prefix), None


def _side_by_side(c: VeroraxConfig, i: int, shapes) -> tuple[PartSpec, PartSpec | None]:
    m, where, prefix = c.layers[i].mixer, f"layers[{i}].mixer", f"l{i}.mix."
    left, right = need(m, "left", where), need(m, "right", where)
    dim = pos_int(left, "dim", where + ".left")
    lp = {"hidden_size": c.width, **head_counts(left, where + ".left"), "key_dim": dim, "value_dim": pos_int(left, "vdim", where + ".left"),
          "scale": number(left, "scale", where + ".left"), "eps": c.eps, "qk_norm": "weighted", "head_temperature": True,
          "window": _window(left, where + ".left"), "output_gate": "head"}
    position = _rotation(left, where + ".left", dim)
    stored = (shapes or {}).get(prefix + "right.w1")
    rank = int(stored[0]) if stored else (pos_int(right, "rank", where + ".right") if "rank" in right else DECAY_RANK)
    rp = {"hidden_size": c.width, "num_heads": pos_int(right, "heads", where + ".right"), "dim": pos_int(right, "dim", where + ".right"),
          "decay_rank": rank, "eps": c.eps}
    return PartSpec("mixer_pair", {
        "hidden_size": c.width, "eps": c.eps, "scales": (number(m, "left_scale", where), number(m, "right_scale", where)),
        "left": {"kind": "gated_attention", "params": lp, "position": {"kind": position.kind, "params": position.params} if position else None},
        "right": {"kind": "delta_rule", "params": rp}}, prefix=prefix), None


_MIXERS = {"latent_attention": _latent, "attention": _differential, "parallel": _side_by_side}


# ---- one function per feed-forward kind
def _dense(c: VeroraxConfig, mlp: Mapping[str, Any], prefix: str) -> PartSpec:
    return PartSpec("gelu_glu", {"hidden_size": c.width, "intermediate_size": pos_int(mlp, "ff", prefix + "mlp")}, prefix=prefix + "mlp.")


def _experts(c: VeroraxConfig, mlp: Mapping[str, Any], prefix: str) -> PartSpec:
    where = prefix + "mlp"
    router = need(mlp, "router", where)
    params = {"hidden_size": c.width, "intermediate_size": pos_int(need(mlp, "expert", where), "ff", where + ".expert"),
              "experts": pos_int(router, "experts", where + ".router"), "top": pos_int(router, "top", where + ".router"),
              "identity": nonneg_int(router, "identity", where + ".router") if "identity" in router else 0, "activation": "silu_glu", "score": "softmax",
              "renormalize": False, "choice_correction": True}
    if params["top"] > params["experts"] + params["identity"]:
        raise ConfigError(f"config.json: {where}.router: {params['top']} of {params['experts'] + params['identity']} experts cannot be chosen")
    return PartSpec("routed_experts", params, prefix=prefix + "mlp.")


_FEED_FORWARDS = {"dense": _dense, "moe": _experts}


def verorax_model_spec(c: VeroraxConfig, shapes: Mapping[str, tuple[int, ...]] | None = None) -> ModelSpec:
    """``shapes``: the checkpoint's tensor shapes (None without a checkpoint); they give the one size config.json leaves out."""
    def norm(name: str) -> PartSpec:
        return PartSpec("rms_norm", {"size": c.width, "eps": c.eps}, prefix=name, names={"weight": ""})

    layers: list[LayerSpec] = []
    index: dict[int, int] = {}     # layer with tensors -> its place among the spec's layers
    for i, layer in enumerate(c.layers):
        if layer.owner != i:
            continue
        p = f"l{i}."
        mixer, position = _MIXERS[layer.type](c, i, shapes)
        ff = _FEED_FORWARDS[layer.mlp["kind"]](c, layer.mlp, p) if layer.mlp is not None else None
        index[i] = len(layers)
        layers.append(LayerSpec(
            mixer=mixer, mixer_norm=norm(p + "norm1"), mixer_post_norm=norm(p + "norm1b"), feed_forward=ff,
            feed_forward_norm=norm(p + "norm2") if ff else None, feed_forward_post_norm=norm(p + "norm2b") if ff else None, position=position,
            block=PartSpec("shifted_sandwich_norm", {"hidden_size": c.width}, prefix=p)))
    return ModelSpec(
        architecture=c.architecture, hidden_size=c.width, vocab_size=c.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": c.width, "scale": 1.0, "whole_stream": True},
                           prefix="embed", names={"weight": ""}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(index[layer.owner]) for layer in c.layers),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": c.vocab, "hidden_size": c.width, "tied": False}, prefix="head", names={"weight": ""}),
        max_positions=MAX_POSITIONS, eos_token_ids=c.eos_token_ids,
        # a layer without a feed-forward may still carry the norms of one
        ignored_tensors=(r"l\d+\.norm2b?",))


VERORAX = register_architecture(Architecture("Verorax", VeroraxConfig.from_dict, verorax_model_spec, shapes_matter=True))

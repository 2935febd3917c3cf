"""The decoder: embedding, a schedule of blocks, final norm, output head. Built from a ModelSpec alone."""

from __future__ import annotations

from typing import Any

import torch

from oxr_inference_b200 import ops
from oxr_inference_b200.cache.plan import CachePlan, make_cache_plan
from oxr_inference_b200.parts.base import (ARRANGEMENTS, EMBEDDINGS, FEED_FORWARDS, HEADS, JOINTS, MIXERS, NORMS, POSITION_ENCODINGS,
                                           Embedding, Head, ParamInfo, Part, Runtime, StepContext)
from oxr_inference_b200.parts.spec import ModelSpec, PartSpec


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding(Embedding):
    """``x = table[ids] * scale`` (oxr_runtime/language.py:155, oxr_runtime/decode_graph.py:75; the reference has no scale).
    ``whole_stream``: the output is the fp32 residual stream itself (for blocks that keep the stream whole) instead of
    activations that the first norm turns into one."""

    def __init__(self, runtime: Runtime, *, vocab_size: int, hidden_size: int, scale: float = 1.0, whole_stream: bool = False):
        self.runtime, self.vocab, self.hidden = runtime, int(vocab_size), int(hidden_size)
        self.scale, self.whole_stream = float(scale), bool(whole_stream)
        self.weight: torch.Tensor | None = None

    def parameters(self) -> dict[str, ParamInfo]:
        return {"weight": ParamInfo((self.vocab, self.hidden))}

    def assign(self, name: str, tensor: torch.Tensor) -> None:
        if name != "weight":
            raise KeyError(name)
        dtype = self.runtime.store_dtype(self.parameters()["weight"], tensor.dtype)
        self.weight = tensor.to(device=self.runtime.device, dtype=dtype).contiguous()

    def forward(self, ids: torch.Tensor) -> torch.Tensor:
        return ops.embedding(ids, self.weight, torch.float32 if self.whole_stream else self.runtime.dtype, self.runtime.status, self.scale)


@HEADS.register("linear_head")
class OutputHead(Head):
    """``logits = h W^T`` in fp32 (oxr_runtime/language.py:158,213-214). ``tied``: W is the embedding table, which
    the reference does not offer (its head is always a tensor of its own). ``scale``: the fp32 logits are multiplied by it. ``softcap`` > 0:
    the logits then become ``softcap * tanh(logits / softcap)``."""

    def __init__(self, runtime: Runtime, embedding: Embedding, *, vocab_size: int, hidden_size: int, tied: bool, scale: float = 1.0,
                 softcap: float = 0.0):
        self.runtime, self.embedding = runtime, embedding
        self.vocab, self.hidden, self.tied, self.scale = int(vocab_size), int(hidden_size), bool(tied), float(scale)
        self.softcap = float(softcap)
        if self.softcap < 0:
            raise ValueError("softcap must not be negative (0 turns it off)")
        self.weight: torch.Tensor | None = None

    def parameters(self) -> dict[str, ParamInfo]:
        return {} if self.tied else {"weight": ParamInfo((self.vocab, self.hidden))}

    def assign(self, name: str, tensor: torch.Tensor) -> None:
        if name != "weight" or self.tied:
            raise KeyError(name)
        dtype = self.runtime.store_dtype(self.parameters()["weight"], tensor.dtype)
        self.weight = tensor.to(device=self.runtime.device, dtype=dtype).contiguous()

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        w = self.embedding.weight if self.tied else self.weight
        logits = ops.linear(h, w, torch.float32)
        if self.scale != 1.0:
            ops.scale_(logits, self.scale)
        return ops.tanh_cap_(logits, self.softcap) if self.softcap > 0 else logits


class DecoderModel:
    def __init__(self, spec: ModelSpec, runtime: Runtime):
        self.spec, self.runtime = spec, runtime
        self._named: dict[str, tuple[Part, str, ParamInfo]] = {}
        self._positions: dict[tuple, Any] = {}

        self.embedding = EMBEDDINGS.build(spec.embedding.kind, runtime, **spec.embedding.params)
        self._register(self.embedding, spec.embedding)

        self.blocks = []
        for layer in spec.layers:
            position = self._position(layer.position)
            mixer = MIXERS.build(layer.mixer.kind, runtime, position, **layer.mixer.params)
            mixer_norm = NORMS.build(layer.mixer_norm.kind, runtime, **layer.mixer_norm.params)
            ff = FEED_FORWARDS.build(layer.feed_forward.kind, runtime, **layer.feed_forward.params) if layer.feed_forward else None
            ff_norm = NORMS.build(layer.feed_forward_norm.kind, runtime, **layer.feed_forward_norm.params) if layer.feed_forward_norm else None
            made = [(mixer, layer.mixer), (mixer_norm, layer.mixer_norm), (ff, layer.feed_forward), (ff_norm, layer.feed_forward_norm)]
            post = {}
            for key, post_spec in (("mixer_post_norm", layer.mixer_post_norm), ("feed_forward_post_norm", layer.feed_forward_post_norm)):
                if post_spec is not None:
                    post[key] = NORMS.build(post_spec.kind, runtime, **post_spec.params)
                    made.append((post[key], post_spec))
            if layer.block is not None:   # an arrangement with parameters and tensors of its own
                block = ARRANGEMENTS.build(layer.block.kind, mixer, mixer_norm, ff, ff_norm, runtime=runtime, **layer.block.params, **post)
                made.append((block, layer.block))
            else:
                block = ARRANGEMENTS.build(layer.arrangement, mixer, mixer_norm, ff, ff_norm, **post)
            self.blocks.append(block)
            for part, part_spec in made:
                if part is not None:
                    self._register(part, part_spec)

        self.joints = []
        for joint_spec in spec.joints:
            self.joints.append(JOINTS.build(joint_spec.kind, runtime, **joint_spec.params))
            self._register(self.joints[-1], joint_spec)

        self.final_norm = NORMS.build(spec.final_norm.kind, runtime, **spec.final_norm.params)
        self._register(self.final_norm, spec.final_norm)
        self.head = HEADS.build(spec.head.kind, runtime, self.embedding, **spec.head.params)
        self._register(self.head, spec.head)

        for i, entry in enumerate(spec.schedule):
            if not 0 <= entry.layer < len(self.blocks):
                raise ValueError(f"schedule entry {i} names layer {entry.layer}; the model has {len(self.blocks)}")
            if entry.joint is not None and not 0 <= entry.joint < len(self.joints):
                raise ValueError(f"schedule entry {i} names joint {entry.joint}; the model has {len(self.joints)}")
        self.schedule = spec.schedule
        self.cache_plan: CachePlan = make_cache_plan(
            [self._cache_need(self.blocks[e.layer]) for e in self.schedule], [e.cache_of for e in self.schedule])
        self.tile_specs = sorted({spec for b in self.blocks for spec in b.mixer.tile_specs()})

    # ---- construction helpers
    @staticmethod
    def _cache_need(block):
        """What one run of a block keeps: its mixer's need, unless the arrangement keeps something of its own beside it."""
        own = getattr(block, "cache_need", None)
        return own() if own is not None else block.mixer.cache_need()

    def _position(self, spec: PartSpec | None):
        if spec is None:
            return None
        key = spec.key()
        if key not in self._positions:
            self._positions[key] = POSITION_ENCODINGS.build(spec.kind, self.runtime, **spec.params)
        return self._positions[key]

    def _register(self, part: Part, spec: PartSpec) -> None:
        for local, info in part.parameters().items():
            name = spec.prefix + spec.names.get(local, local)
            if name in self._named:
                raise ValueError(f"two parts claim the tensor {name!r}")
            self._named[name] = (part, local, info)

    def named_parameters(self) -> dict[str, tuple[Part, str, ParamInfo]]:
        """Checkpoint name -> (part that takes it, the part's local name, shape and kind)."""
        return dict(self._named)

    def parts(self) -> list[Part]:
        seen, out = set(), []
        for part, _, _ in self._named.values():
            if id(part) not in seen:
                seen.add(id(part))
                out.append(part)
        return out

    def head_dims(self) -> tuple[int, ...]:
        """Head sizes whose per-size attention library this model's mixers run."""
        return tuple(sorted({d for b in self.blocks for d in b.mixer.kernel_head_dims()}))

    # ---- the forward pass of one step
    def step(self, ctx: StepContext, cache) -> torch.Tensor:
        """Run the step's tokens through every scheduled block; fp32 logits ``[len(ctx.logit_rows), vocab]``."""
        ctx.shared.clear()
        x = self.embedding.forward(ctx.token_ids)
        residual = None
        first = None
        if self.joints:
            # joints read the embedding's output again later: blocks that keep the stream whole write into their own copy
            first, x = x, x.clone()
        for pos, entry in enumerate(self.schedule):
            block = self.blocks[entry.layer]
            if entry.joint is not None:
                if residual is None:
                    x, residual = None, x
                elif x is not None:
                    raise ValueError("a joint needs the stream whole: the block before it left an output that is not yet added")
                residual = self.joints[entry.joint].forward(residual, first, entry.joint_arg, ctx)
            # a block may leave its last projection to the next block's norm, if both sides say that they can
            after = self.blocks[self.schedule[pos + 1].layer] if pos + 1 < len(self.schedule) else None
            keeps_add = getattr(block, "keeps_add_for", None)
            if (getattr(block, "supports_deferred", False) and getattr(after, "accepts_deferred_input", False)) or (
                    keeps_add is not None and keeps_add(after) and self.schedule[pos + 1].joint is None):
                x, residual = block.forward(x, residual, ctx, cache.layer_cache(pos, ctx), defer_output=True)
            else:
                x, residual = block.forward(x, residual, ctx, cache.layer_cache(pos, ctx))
        if ctx.logit_rows.numel() == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=self.runtime.device)
        if x is None:   # the blocks kept the stream whole
            h = self.final_norm.stream_rows(residual, ctx.logit_rows)
        else:
            h = self.final_norm.forward_rows(x, residual, ctx.logit_rows)
        return self.head.forward(h)

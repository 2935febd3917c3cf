"""Differential attention: two softmax maps per head over the same values, one subtracted from the other."""

from __future__ import annotations

import torch

from oxr_inference_b200 import ops
from oxr_inference_b200.parts.base import MIXERS, LayerCache, Mixer, PagedKVNeed, ParamInfo, PositionEncoding, Runtime, StepContext
from oxr_inference_b200.parts.linear import StackedLinear


@MIXERS.register("differential_attention")
class DifferentialAttention(Mixer):
    """``q, k, v = h W^T`` (+ ``q.b``, ``k.b``, ``v.b`` with ``biases``), where every query and key head is a pair ``[map 1 | map 2]`` of ``dim`` entries each and
    head h reads key/value head ``h // (heads / kv_heads)``. Map m is causal softmax attention with scores ``q_m . k_m * scale`` (``window`` > 0: the
    last ``window`` keys only) over the head's values of ``value_dim`` entries. With the two maps' outputs a1, a2 and one number per layer ``lambda =
    exp(sum lq1 lk1) - exp(sum lq2 lk2) + diff``:

        o = a1 - lambda a2        o <- o / sqrt(mean(o^2) + eps) * (1 - diff)

    over each head's entries, then ``W_o``. No rotation.

    Both maps run as heads of ordinary grouped-query attention over one cached key row per key head: the queries ``[q1 | 0]`` and ``[0 | q2]``
    over rows ``[k1 | k2]``, so keys and values are kept and read once and the engine's attention kernels serve as they are. In bfloat16 keys
    and values stand in the cache at one size (the larger of ``2 dim`` and ``value_dim``, whole multiples of 16; what is added stays zero), which is
    what the tensor-core kernels take."""

    def __init__(self, runtime: Runtime, position: PositionEncoding | None, *, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int,
                 value_dim: int, scale: float, diff: float, eps: float, window: int = 0, biases: bool = False):
        if position is not None:
            raise ValueError("differential_attention takes no position encoding")
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} KV heads")
        self.runtime = runtime
        self.hidden, self.H, self.G, self.D, self.DV = int(hidden_size), int(num_heads), int(num_kv_heads), int(dim), int(value_dim)
        self.scale, self.diff, self.eps, self.window, self.biases = float(scale), float(diff), float(eps), int(window), bool(biases)
        self.proj = StackedLinear(runtime, self.hidden, {"q": 2 * self.H * self.D, "k": 2 * self.G * self.D, "v": self.G * self.DV})
        self.out = StackedLinear(runtime, self.H * self.DV, {"o": self.hidden})
        size = (max(2 * self.D, self.DV) + 15) // 16 * 16
        self.tiled = ops.tiled_attention_takes(size, size, runtime.dtype)
        self.width, self.value_width = (size, size) if self.tiled else (2 * self.D, self.DV)
        self.vectors: dict[str, torch.Tensor] = {}
        self.bias: torch.Tensor | None = None
        self.lam: torch.Tensor | None = None

    def _vector_shapes(self) -> dict[str, tuple[int, ...]]:
        out = {name: (self.D,) for name in ("lq1", "lk1", "lq2", "lk2")}
        if self.biases:
            out.update({name + ".b": (n,) for name, n in self.proj.outs.items()})
        return out

    def parameters(self) -> dict[str, ParamInfo]:
        return {**self.proj.parameters(), **self.out.parameters(),
                **{name: ParamInfo(shape, role="vector") for name, shape in self._vector_shapes().items()}}

    def assign(self, name: str, tensor: torch.Tensor) -> None:
        if name in self.proj.outs:
            self.proj.assign(name, tensor)
        elif name in self.out.outs:
            self.out.assign(name, tensor)
        elif name in self._vector_shapes():
            self.vectors[name] = tensor.to(device=self.runtime.device, dtype=torch.float32).contiguous()
        else:
            raise KeyError(name)

    def finish_loading(self) -> None:
        v = {name: t.double() for name, t in self.vectors.items()}
        self.lam = (torch.exp((v["lq1"] * v["lk1"]).sum()) - torch.exp((v["lq2"] * v["lk2"]).sum()) + self.diff).float().reshape(1).contiguous()
        if self.biases:
            self.bias = torch.cat([self.vectors[name + ".b"] for name in self.proj.outs]).contiguous()

    def cache_need(self) -> PagedKVNeed:
        # keys and values of one size: the need of plain grouped-query attention, whose pools get TMA maps
        return PagedKVNeed(self.G, self.width, self.window, value_dim=None if self.value_width == self.width else self.value_width)

    def kernel_head_dims(self) -> tuple[int, ...]:
        return (self.width,) if self.tiled else ()

    def tile_specs(self) -> list[tuple[int, int, int]]:
        return ops.attention_tile_specs(2 * self.H, self.G, self.width, self.runtime.dtype, self.runtime.page_size) if self.tiled else []

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        group = cache.group
        k_pool, v_pool = group.k_pool[cache.layer_in_group], group.v_pool[cache.layer_in_group]
        n = ctx.n_tokens
        proj = self.proj(h)
        if proj.dtype != k_pool.dtype:
            proj = ops.cast(proj, k_pool.dtype)
        q = ops.diff_prep(proj, num_heads=self.H, num_kv_heads=self.G, dim=self.D, value_dim=self.DV, width=self.width, bias=self.bias, k_pool=k_pool,
                          v_pool=v_pool, slots=group.slots if cache.store else ctx.no_store_slots, status=ctx.status)
        if self.tiled:
            o = ops.paged_attention(q.view(n, 2 * self.H, self.width), k_pool, v_pool, tiles=ctx.tiles, cu_q=ctx.cu_q, ctx_lens=ctx.ctx_lens,
                                    block_table=group.block_table, page_size=group.page_size, scale=self.scale, window=self.window,
                                    kv_len_bound=ctx.kv_len_bound, status=ctx.status, kv_maps=group.kv_maps, layer_in_pool=cache.layer_in_group,
                                    uneven=ctx.uneven)
        else:
            o = ops.attention_rows(q, 2 * self.H, k_pool, v_pool, value_dim=self.DV, positions=ctx.positions, req_of_token=ctx.req_of_token,
                                   block_table=group.block_table, scale=self.scale, window=self.window, status=ctx.status).view(n, 2 * self.H, self.DV)
        return self.out(ops.diff_combine(o, self.H, self.DV, self.lam, self.eps, 1.0 - self.diff))

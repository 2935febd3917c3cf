"""A generalized delta rule: a recurrence that takes out along a key what it holds there before it adds, with a decay per key channel."""

from __future__ import annotations

import math

import torch

from oxr_inference_b200 import ops
from oxr_inference_b200.parts.base import MIXERS, LayerCache, Mixer, ParamInfo, PositionEncoding, Runtime, StateNeed, StepContext
from oxr_inference_b200.parts.linear import StackedLinear


@MIXERS.register("delta_rule")
class DeltaRule(Mixer):
    """``r = W_r h``, ``k = W_k h``, ``v = W_v h`` (``heads x dim`` each); per head and key channel a decay ``w = exp(-rate * sigmoid(W_w2 tanh(W_w1 h) + w0))``
    (a low-rank map; ``rate`` is exp(-1/2) by default, so that no channel keeps less than exp(-0.61) of what it holds) and a removal rate
    ``a = sigmoid(W_a h + a.b)``. Per head, with the unit key ``u = k / sqrt(sum k^2 + length_eps)`` and S zero at a sequence's start:

        S_t = diag(w_t) S_(t-1) - (a_t * u_t) (u_t^T S_(t-1)) + k_t v_t^T        o_t = S_t^T r_t

    with everything on the right taken from S_(t-1). Then each head's o is divided by its root mean square, the heads side by side are multiplied by ``norm``
    (one weight per head and entry) and by ``sigmoid(W_g h)``, then ``W_o``. r, k, v and the gate are one product; ``W_a`` and ``W_w1`` are a second
    one whose result stays fp32, like that of ``W_w2`` and everything else that enters the recurrence behind the projections. Per request the
    mixer keeps one fp32 state row: S transposed, ``[heads, values, keys]``; zero for a new request, carried from step to step whatever the
    cut."""

    def __init__(self, runtime: Runtime, position: PositionEncoding | None, *, hidden_size: int, num_heads: int, dim: int, decay_rank: int, eps: float,
                 rate: float = math.exp(-0.5), length_eps: float = 1e-6):
        if position is not None:
            raise ValueError("delta_rule takes no position encoding")
        if dim > 256:
            raise ValueError(f"the recurrence kernel keeps heads of up to 256 entries, got {dim}")
        self.runtime = runtime
        self.hidden, self.H, self.D, self.rank = int(hidden_size), int(num_heads), int(dim), int(decay_rank)
        self.eps, self.rate, self.length_eps = float(eps), float(rate), float(length_eps)
        self.inner = self.H * self.D
        self.in_proj = StackedLinear(runtime, self.hidden, {"r": self.inner, "k": self.inner, "v": self.inner, "g": self.inner})
        self.rates = StackedLinear(runtime, self.hidden, {"a": self.inner, "w1": self.rank})
        self.decay = StackedLinear(runtime, self.rank, {"w2": self.inner})
        self.out = StackedLinear(runtime, self.inner, {"o": self.hidden})
        self.vectors: dict[str, torch.Tensor] = {}

    _VECTORS = ("w0", "a.b", "norm")

    def parameters(self) -> dict[str, ParamInfo]:
        return {**self.in_proj.parameters(), **self.rates.parameters(), **self.decay.parameters(), **self.out.parameters(),
                "w0": ParamInfo((self.inner,), role="vector"), "a.b": ParamInfo((self.inner,), role="vector"),
                "norm": ParamInfo((self.inner,), init="around_one", role="vector")}

    def assign(self, name: str, tensor: torch.Tensor) -> None:
        for stack in (self.in_proj, self.rates, self.decay, self.out):
            if name in stack.outs:
                stack.assign(name, tensor)
                return
        if name not in self._VECTORS:
            raise KeyError(name)
        self.vectors[name] = tensor.to(device=self.runtime.device, dtype=torch.float32).contiguous()

    def cache_need(self) -> StateNeed:
        return StateNeed((self.inner * self.D,), torch.float32)

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        v = self.vectors
        proj = self.in_proj(h)                              # [tokens, r | k | v | g]
        rates = self.rates(h, torch.float32)                # [tokens, a | w1], kept in fp32
        z = self.decay(ops.tanh_cols(rates, self.inner, self.rank, h.dtype), torch.float32)
        o = ops.delta_scan(proj, 0, self.inner, 2 * self.inner, z, v["w0"], rates, v["a.b"], heads=self.H, key_dim=self.D, value_dim=self.D,
                           rate=self.rate, len_eps=self.length_eps, state=cache.state, cu_q=ctx.cu_q, state_slots=ctx.state_slots,
                           n_requests=ctx.n_requests, single_tokens=ctx.single_tokens)
        return self.out(ops.head_norm_gate(o, proj, 3 * self.inner, v["norm"], self.H, self.eps))

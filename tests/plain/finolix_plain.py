"""A plain, slow statement of the Finolix decoder: one function per mechanism, whole sequences at once, no cache.

Shares no code with the engine. Everything runs on the host in one floating-point type (float64 by default), so it is the
yardstick for both the 16-bit and the 32-bit engine. The network: a token embedding copied into several residual streams; a list of layers, each
a mixer and (unless the layer has none) a feed-forward, where every sublayer reads the norm of a weighted sum of the streams and its result,
scaled entry by entry, goes to every stream with a weight of that stream's while the streams are mixed by a small matrix; then the sum of the
streams, an RMS norm and an untied output head. Norm weights of the stream's norms are stored around zero. A layer may run with another layer's
tensors. Two mixers: attention over a compressed row per token, with queries that pass a latent of their own, a rotation of neighbouring
entries whose frequencies follow a ramp, a window and a sink per head; and causal grouped-query attention with q/k norm, a half-split rotation
of part of each head, and one gate per head. Feed-forwards: a two-matrix layer with the square of relu, or routed SiLU-gated experts weighted by
the softmax over the chosen logits.
"""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch
from safetensors import safe_open


def read_model(folder: str | Path, dtype: torch.dtype = torch.float64):
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    w = {}
    with safe_open(str(folder / "model.safetensors"), framework="pt", device="cpu") as f:
        for name in f.keys():  # noqa: SIM118
            t = f.get_tensor(name)
            w[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, w


# ------------------------------------------------------------------------------------------------ small pieces
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * (1.0 + weight)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def heads_of(x: torch.Tensor, n: int) -> torch.Tensor:
    return x.reshape(x.shape[0], n, -1)


# ------------------------------------------------------------------------------------------------ rotation
def ramp_frequencies(dims: int, base: float, scaling: dict | None) -> tuple[list[float], float]:
    """One frequency per pair and the factor on cos and sin: ``base^(-2i/dims)``, slowed down towards 1/factor of itself for the pairs that turn
    few times within ``original`` positions."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def dim_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / factor * ramp + f[i] * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, freq: list[float], magnitude: float, neighbours: bool) -> torch.Tensor:
    """x: [T, heads, D]. Pair i is entries 2i and 2i + 1 (``neighbours``) or i and i + the number of pairs; it turns by position * freq[i] and is
    stretched by ``magnitude``; the other entries stay."""
    n = len(freq)
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(freq):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + n)
        c, s = (torch.cos(pos * f) * magnitude).to(x.dtype)[:, None], (torch.sin(pos * f) * magnitude).to(x.dtype)[:, None]
        u, v = x[:, :, a], x[:, :, b]
        out[:, :, a] = u * c - v * s
        out[:, :, b] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------ softmax attention
def visible(T: int, window: int = 0) -> torch.Tensor:
    """[T, T] bool: query i sees key j <= i; with a window only if i - j < window."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i - j < window) if window > 0 else seen


def attend(scores: torch.Tensor, seen: torch.Tensor, v: torch.Tensor, sink: torch.Tensor | None = None) -> torch.Tensor:
    """scores [T, T] -> weights over what is seen -> weighted sum of v [T, DV]. A sink is one more score in the denominator, without a value."""
    s = scores.masked_fill(~seen, -math.inf)
    if sink is None:
        return torch.softmax(s, -1) @ v
    s = torch.cat([s, sink.reshape(1, 1).expand(s.shape[0], 1)], 1)
    return torch.softmax(s, -1)[:, :-1] @ v


# ------------------------------------------------------------------------------------------------ the mixers
def latent_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """Keys and values are per-head maps of one normed latent per token; a rotated key part is shared by the heads."""
    T, H, D, R, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = heads_of((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T, H)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :L], eps) * w[p + "dkv.norm"]
    freq, magnitude = ramp_frequencies(m["rot"]["dims"], float(m["rot"]["base"]), m["rot"].get("scaling"))
    q_turned = rotate(q[:, :, D:], freq, magnitude, True)
    k_turned = rotate(down[:, None, L:L + R], freq, magnitude, True)[:, 0]
    k = heads_of(c @ w[p + "uk"].T, H)
    v = heads_of(c @ w[p + "uv"].T, H)
    seen = visible(T, m["mask"]["size"])
    o = [attend((q[:, i, :D] @ k[:, i].T + q_turned[:, i] @ k_turned.T) * m["scale"], seen, v[:, i], w[p + "sink"][i]) for i in range(H)]
    return torch.cat(o, -1) @ w[p + "o"].T


def gated_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    freq, magnitude = ramp_frequencies(m["rot"]["dims"], float(m["rot"]["base"]), None)
    q = rotate(rms(heads_of(h @ w[p + "q"].T, H), eps) * w[p + "q.norm"], freq, magnitude, False)
    k = rotate(rms(heads_of(h @ w[p + "k"].T, G), eps) * w[p + "k.norm"], freq, magnitude, False)
    v = heads_of(h @ w[p + "v"].T, G)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    seen = visible(T)
    o = [attend((q[:, i] @ k[:, i // (H // G)].T) * m["scale"], seen, v[:, i // (H // G)]) * gate[:, i:i + 1] for i in range(H)]
    return torch.cat(o, -1) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "attention": gated_attention}


# ------------------------------------------------------------------------------------------------ feed-forwards
def squared_relu(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return (torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2) @ w[p + "down"].T


def silu_unit(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router_logits(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return h @ w[p + "router"].T + w[p + "router.b"]


def choice_margin(z: torch.Tensor, top: int) -> torch.Tensor:
    """How far the last chosen logit is above the best one not chosen (inf when all are chosen)."""
    s = torch.sort(z, dim=-1, descending=True).values
    if top >= s.shape[1]:
        return torch.full((s.shape[0],), math.inf, dtype=z.dtype)
    return s[:, top - 1] - s[:, top]


def routed_experts(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    z = router_logits(h, w, p)
    best = torch.topk(z, mlp["router"]["top"], dim=-1)
    share = torch.softmax(best.values, -1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j, e in enumerate(best.indices[t].tolist()):
            out[t] += share[t, j] * silu_unit(h[t][None], w, f"{p}e{e}.")[0]
    return out


def feed_forward(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return squared_relu(h, w, p)
    if mlp["kind"] == "moe":
        return routed_experts(h, w, p, mlp)
    raise ValueError(mlp["kind"])


# ------------------------------------------------------------------------------------------------ streams
def read_streams(x: torch.Tensor, weights: torch.Tensor) -> torch.Tensor:
    """x [streams, T, width] -> what a sublayer reads (before its norm)."""
    return (weights[:, None, None] * x).sum(0)


def write_streams(x: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """New stream t = sum over s of mix[s, t] * old stream s, plus out[t] * y."""
    return torch.stack([sum(mix[s, t] * x[s] for s in range(x.shape[0])) + out[t] * y for t in range(x.shape[0])])


# ------------------------------------------------------------------------------------------------ the model
def owner_of(layers: list[dict], i: int) -> int:
    """The layer whose tensors layer i runs with."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg: dict, w: dict, tokens: list[int], streams: list | None = None, margins: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence. ``streams`` collects the sum of the streams after every layer, ``margins`` the routers' margins."""
    eps = float(cfg["norm"]["eps"])
    x = torch.stack([w["embed"][torch.tensor(tokens, dtype=torch.long)]] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner_of(cfg['layers'], i)}."
        h = norm_around_zero(read_streams(x, w[p + "hc1.in"]), w[p + "norm1"], eps)
        y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps) * w[p + "ls1"]
        x = write_streams(x, w[p + "hc1.mix"], w[p + "hc1.out"], y)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm_around_zero(read_streams(x, w[p + "hc2.in"]), w[p + "norm2"], eps)
            if margins is not None and mlp["kind"] == "moe":
                margins.append(choice_margin(router_logits(h, w, p + "mlp."), mlp["router"]["top"]))
            y = feed_forward(h, w, p + "mlp.", mlp) * w[p + "ls2"]
            x = write_streams(x, w[p + "hc2.mix"], w[p + "hc2.out"], y)
        if streams is not None:
            streams.append(x.sum(0))
    return norm_around_zero(x.sum(0), w["final.norm"], eps) @ w["head"].T


def greedy(cfg: dict, w: dict, prompt: list[int], n: int) -> tuple[list[int], list[float]]:
    """``n`` greedy tokens after ``prompt`` and, for each, how far its logit stood above the runner-up's."""
    tokens, gaps = list(prompt), []
    for _ in range(n):
        last = forward(cfg, w, tokens)[-1]
        best = torch.topk(last, 2).values
        gaps.append(float(best[0] - best[1]))
        tokens.append(int(last.argmax()))
    return tokens[len(prompt):], gaps

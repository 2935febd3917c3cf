"""A plain, slow statement of the Verorax decoder: one function per mechanism, whole sequences at once, no cache.

Shares no code with the engine. Everything runs on the host in one floating-point type (float64 by default), so it is the
yardstick for both the 16-bit and the 32-bit engine. The network: a token embedding; a list of layers, each ``x += norm1b(mixer(g))``
with ``g`` the normed stream ``norm1(x)`` blended with the previous token's, and then ``x += norm2b(ff(norm2(x)))``; a final RMS norm; an
untied output head. A layer may run with another layer's tensors. Three mixers: attention over a compressed row per token, with queries
that pass a low-rank latent of their own; differential attention (two softmax maps per head over the same values, one subtracted from the
other) with biases and a window; and a pair, windowed attention with q/k norm, rotation, a temperature and a gate per head beside a
delta-rule recurrence with a decay per key channel. Feed-forwards: a GELU-gated layer, or routed SiLU-gated experts some of which return
their input.
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


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def heads_of(x: torch.Tensor, n: int) -> torch.Tensor:
    return x.reshape(x.shape[0], n, -1)


def token_shift(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """Every entry moves the share ``mu`` of the way to the previous token's entry (zero before the first token)."""
    before = torch.zeros_like(h)
    before[1:] = h[:-1]
    return h + (before - h) * mu


# ------------------------------------------------------------------------------------------------ rotation
def rotate_halves(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x: [T, heads, D]. Entry i < dims / 2 is paired with entry i + dims / 2; the pair turns by position * base^(-2i/dims); entries
    from dims on stay."""
    n = dims // 2
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(n):
        a = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + n]
        out[:, :, i] = u * c - v * s
        out[:, :, i + n] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------ softmax attention
def visible(T: int, window: int = 0) -> torch.Tensor:
    """[T, T] bool: query i sees key j <= i; with a window only if i - j < window."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i - j < window) if window > 0 else seen


def attend(scores: torch.Tensor, seen: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
    """scores [T, T] -> softmax over what is seen -> weighted sum of v [T, DV]."""
    return torch.softmax(scores.masked_fill(~seen, -math.inf), -1) @ v


# ------------------------------------------------------------------------------------------------ the mixers
def latent_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """Keys and values are per-head maps of one normed latent per token; a rotated key part is shared by the heads."""
    T, H, D, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    L = m["kv_rank"]
    q = heads_of((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T, H)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :L], eps) * w[p + "dkv.norm"]
    base = float(m["rot"]["base"])
    q_turned = rotate_halves(q[:, :, D:], R, base)
    k_turned = rotate_halves(down[:, None, L:], R, base)[:, 0]
    k = heads_of(c @ w[p + "uk"].T, H)
    v = heads_of(c @ w[p + "uv"].T, H)
    seen = visible(T)
    o = [attend((q[:, i, :D] @ k[:, i].T + q_turned[:, i] @ k_turned.T) * m["scale"], seen, v[:, i]) for i in range(H)]
    return torch.cat(o, -1) @ w[p + "o"].T


def map_weight(w: dict, p: str, diff: float) -> torch.Tensor:
    """How much of the second map is subtracted: one number per layer."""
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def differential_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, 2, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, 2, D)
    v = heads_of(h @ w[p + "v"].T + w[p + "v.b"], G)
    seen = visible(T, m["mask"]["size"])
    lam = map_weight(w, p, m["diff"])
    out = []
    for i in range(H):
        g = i // (H // G)
        one, two = (attend((q[:, i, j] @ k[:, g, j].T) * m["scale"], seen, v[:, g]) for j in (0, 1))
        out.append(rms(one - lam * two, eps) * (1.0 - m["diff"]))
    return torch.cat(out, -1) @ w[p + "o"].T


def gated_window_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """The pair's left side."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms(heads_of(h @ w[p + "q"].T, H), eps) * w[p + "q.norm"]
    k = rms(heads_of(h @ w[p + "k"].T, G), eps) * w[p + "k.norm"]
    v = heads_of(h @ w[p + "v"].T, G)
    rot = m["rot"]
    q, k = rotate_halves(q, rot["dims"], float(rot["base"])), rotate_halves(k, rot["dims"], float(rot["base"]))
    seen = visible(T, m["mask"]["size"])
    gate = torch.sigmoid(h @ w[p + "g"].T)
    out = []
    for i in range(H):
        g = i // (H // G)
        out.append(attend((q[:, i] @ k[:, g].T) * m["scale"] * w[p + "temp"][i], seen, v[:, g]) * gate[:, i:i + 1])
    return torch.cat(out, -1) @ w[p + "o"].T


def delta_rule(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, rate: torch.Tensor) -> torch.Tensor:
    """All [T, H, D]. Per head, S [D keys, D values] from zero: with u the unit key, what the state holds along u is taken out at
    the rate of each key channel while every key channel decays (both from the old state), k v^T is added, and S^T r is read."""
    T, H, D = k.shape
    unit = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    S = torch.zeros(H, D, v.shape[2], dtype=k.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        held = torch.einsum("hk,hkv->hv", unit[t], S)
        S = decay[t][:, :, None] * S - (rate[t] * unit[t])[:, :, None] * held[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, r[t])
    return o


def delta_mixer(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """The pair's right side."""
    H = m["heads"]
    r, k, v = (heads_of(h @ w[p + n].T, H) for n in ("r", "k", "v"))
    z = torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = heads_of(torch.exp(-math.exp(-0.5) * torch.sigmoid(z)), H)
    rate = heads_of(torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"]), H)
    o = rms(delta_rule(r, k, v, decay, rate), eps).reshape(h.shape[0], -1)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    return (m["left_scale"] * gated_window_attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * delta_mixer(h, w, p + "right.", m["right"], eps))


MIXERS = {"latent_attention": latent_attention, "attention": differential_attention, "parallel": side_by_side}


# ------------------------------------------------------------------------------------------------ feed-forwards
def gated_unit(h: torch.Tensor, w: dict, p: str, act) -> torch.Tensor:
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router_scores(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return torch.softmax(h @ w[p + "router"].T, -1)


def choose(scores: torch.Tensor, correction: torch.Tensor, top: int) -> torch.Tensor:
    return torch.topk(scores + correction, top, dim=-1).indices


def choice_margin(scores: torch.Tensor, correction: torch.Tensor, top: int) -> torch.Tensor:
    """How far the last chosen choice score is above the best one not chosen (inf when all are chosen)."""
    s = torch.sort(scores + correction, dim=-1, descending=True).values
    if top >= s.shape[1]:
        return torch.full((s.shape[0],), math.inf, dtype=scores.dtype)
    return s[:, top - 1] - s[:, top]


def routed_experts(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    """Each token runs ``top`` of ``experts`` gated units and ``identity`` experts behind them that return the input."""
    r = mlp["router"]
    s = router_scores(h, w, p)
    ids = choose(s, w[p + "correction"], r["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in ids[t].tolist():
            y = gated_unit(h[t][None], w, f"{p}e{e}.", silu)[0] if e < r["experts"] else h[t]
            out[t] += s[t, e] * y
    return out


def feed_forward(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return gated_unit(h, w, p, gelu_tanh)
    if mlp["kind"] == "moe":
        return routed_experts(h, w, p, mlp)
    raise ValueError(mlp["kind"])


# ------------------------------------------------------------------------------------------------ the model
def owner_of(layers: list[dict], i: int) -> int:
    """The layer whose tensors layer i runs with."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg: dict, w: dict, tokens: list[int], streams: list | None = None, margins: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence. ``streams`` collects the stream after every layer, ``margins`` the routers' margins."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner_of(cfg['layers'], i)}."
        h = token_shift(rms(x, eps) * w[p + "norm1"], w[p + "shift"])
        x = x + rms(MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps), eps) * w[p + "norm1b"]
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms(x, eps) * w[p + "norm2"]
            if margins is not None and mlp["kind"] == "moe":
                margins.append(choice_margin(router_scores(h, w, p + "mlp."), w[p + "mlp.correction"], mlp["router"]["top"]))
            x = x + rms(feed_forward(h, w, p + "mlp.", mlp), eps) * w[p + "norm2b"]
        if streams is not None:
            streams.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T


def greedy(cfg: dict, w: dict, prompt: list[int], n: int) -> tuple[list[int], list[float]]:
    """``n`` greedy tokens after ``prompt`` and, for each, how far its logit stood above the runner-up's."""
    tokens, gaps = list(prompt), []
    for _ in range(n):
        last = forward(cfg, w, tokens)[-1]
        best = torch.topk(last, 2).values
        gaps.append(float(best[0] - best[1]))
        tokens.append(int(last.argmax()))
    return tokens[len(prompt):], gaps

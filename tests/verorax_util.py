"""Small Verorax configurations and model folders for the tests: sizes unlike any real model's, values that differ where a coincidence
(heads == kv_heads, key size == value size, all entries rotated, top == 1, equal scales, a window that covers everything) would hide a fault,
and weights reshaped so that faults show."""

from __future__ import annotations

import json
from pathlib import Path

import torch


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=5, identity=2, top=3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}


def latent(heads=3, dim=12, rot_dim=8, vdim=20, kv_rank=24, q_rank=28, base=90.0, scale=0.5, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "rot": {"dims": rot_dim, "base": base}, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "scale": scale}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def differential(heads=4, kv_heads=2, dim=10, vdim=24, size=9, diff=0.35, scale=0.6, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": scale, "mask": {"size": size}}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def paired(heads=4, kv_heads=2, dim=16, vdim=24, size=11, rot=12, base=70.0, scale=0.4, r_heads=3, r_dim=12, rank=5, left_scale=0.9, right_scale=0.4,
           mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": {"dims": rot, "base": base}, "scale": scale}
    m = {"left": left, "left_scale": left_scale, "right": {"heads": r_heads, "dim": r_dim, "rank": rank}, "right_scale": right_scale}
    return {"type": "parallel", "mixer": m, "mlp": mlp}


def again(layers, j):
    """Layer j once more: the same entry, running with layer j's tensors."""
    return {**layers[j], "weights_of": j}


def model_config(layers, width=52, vocab=127, eps=1e-5):
    return {"architecture": "Verorax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# Whole models that differ in every size and option.
_A = [latent(mlp=dense()), differential(mlp=moe()), paired(mlp=dense(ff=44)), differential(heads=2, kv_heads=2, dim=8, vdim=8, size=4, diff=0.7)]
MODEL_A = model_config([*_A, again(_A, 1), again(_A, 2), latent(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=16, q_rank=12, mlp=moe(ff=16, experts=3, identity=4, top=2))])
_B = [paired(heads=2, kv_heads=1, dim=32, vdim=32, size=20, rot=32, base=1e4, r_heads=1, r_dim=40, rank=3, left_scale=0.3, right_scale=1.2,
             mlp=moe(ff=8, experts=9, identity=3, top=4)),
      latent(heads=5, dim=16, rot_dim=12, vdim=8, kv_rank=36, q_rank=20, base=1e3, scale=0.3, mlp=dense(ff=72)),
      differential(heads=6, kv_heads=3, dim=16, vdim=32, size=7, diff=0.2, scale=0.5),
      paired(heads=3, kv_heads=3, dim=48, vdim=40, size=33, rot=6, base=9.0, r_heads=4, r_dim=70, rank=9, mlp=dense(ff=24))]
MODEL_B = model_config([*_B, again(_B, 0), latent(heads=1, dim=24, rot_dim=2, vdim=16, kv_rank=8, q_rank=40)], width=64, vocab=200, eps=1e-6)
# every attention layer has sizes that the tensor-core kernels take in bfloat16, and its only router stands in the last layer, where a choice
# that a rounding step turns over spoils one row and no later one
_C = [latent(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=48, q_rank=64, base=500.0, scale=0.2, mlp=dense(ff=48)),
      differential(heads=6, kv_heads=2, dim=32, vdim=64, size=33, diff=0.45, scale=0.3, mlp=dense(ff=32)),
      paired(heads=4, kv_heads=1, dim=128, vdim=128, size=50, rot=64, base=1e3, scale=0.1, r_heads=2, r_dim=64, rank=8, mlp=dense(ff=40))]
MODEL_C = model_config([*_C, again(_C, 2), differential(heads=4, kv_heads=4, dim=16, vdim=48, size=17, diff=0.1, scale=0.4), again(_C, 0),
                        latent(heads=8, dim=64, rot_dim=32, vdim=64, kv_rank=96, q_rank=32, base=1e4, scale=0.15, mlp=moe(ff=32, experts=4, identity=2, top=3))],
                       width=72, vocab=150)


def make_folder(tmp: Path, config: dict, name: str, seed: int = 0, sharpen: float = 2.0, strength: float = 1.0) -> Path:
    """A model folder with random bfloat16 weights, then reshaped so that faults show: queries and keys are scaled up for peaked attention (a
    lost, doubled or wrongly placed key changes the output), biases and the maps' difference get a visible size, temperatures differ, the
    shifts differ from entry to entry, the decay's bias keeps the state alive over many tokens and the removal rates spread, the routers' scores
    and corrections are spread out, gates and experts leave their linear stretch. ``strength`` < 1 scales all of that down towards plain
    random weights, for 16-bit runs of deep models, where every factor here also multiplies what a rounding step does."""
    from safetensors.torch import load_file, save_file

    from oxr_inference_b200.weights import write_random_model

    def by(factor: float) -> float:
        return 1.0 + (factor - 1.0) * strength

    folder = write_random_model(config, tmp / name, seed, dtype="bfloat16", std=0.06)
    path = folder / "model.safetensors"
    tensors = load_file(str(path))
    for k, t in tensors.items():
        f = t.float()
        if k.endswith((".q.norm", ".k.norm", ".dq.norm", ".dkv.norm")):
            f = f * by(sharpen) ** 0.5
        elif k.endswith((".uq", ".uk", ".dkv", ".mix.q", ".mix.k")):
            f = f * by(3)
        elif k.endswith((".q.b", ".k.b", ".v.b")):
            f = f * by(8)
        elif k.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            f = f * by(4)
        elif k.endswith(".temp"):
            f = 1.0 + f * 8
        elif k.endswith(".shift"):
            f = 0.4 + f * 6
        elif k.endswith(".w0"):
            f = f * 20 - 3.0
        elif k.endswith((".w1", ".w2", ".right.a", ".a.b")):
            f = f * by(5)
        elif k.endswith(".router"):
            f = f * by(5)
        elif k.endswith(".correction"):
            f = f * 1.5
        elif k.endswith((".gate", ".up")) and ".mlp." in k:
            f = f * by(4)
        elif k.endswith((".left.g", ".right.g")):
            f = f * by(5)
        elif k.endswith(("head", "embed")):
            f = f * by(4)
        tensors[k] = f.to(t.dtype)
    save_file(tensors, str(path), metadata={"format": "pt"})
    (folder / "config.json").write_text(json.dumps(config, indent=1))
    return folder


def tokens(config: dict, n: int, seed: int) -> list[int]:
    g = torch.Generator().manual_seed(seed * 104729 + n)
    return torch.randint(0, config["vocab"], (n,), generator=g).tolist()


_cache: dict = {}


def plain_logits(folder: Path, ids: list[int]) -> torch.Tensor:
    from plain import verorax_plain as VP

    key = (str(folder), tuple(ids))
    if key not in _cache:
        if str(folder) not in _cache:
            _cache[str(folder)] = VP.read_model(folder, torch.float64)
        cfg, w = _cache[str(folder)]
        margins: list = []
        _cache[key] = VP.forward(cfg, w, ids, margins=margins).float()
        _cache[("margin",) + key] = torch.stack(margins).min(0).values.float() if margins else torch.full((len(ids),), float("inf"))
    return _cache[key]


def router_margins(folder: Path, ids: list[int]) -> torch.Tensor:
    """Per position, the smallest margin by which any layer's router decided (``inf`` without routers)."""
    plain_logits(folder, ids)
    return _cache[("margin", str(folder), tuple(ids))]

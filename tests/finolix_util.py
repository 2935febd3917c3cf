"""Small Finolix configurations and model folders for the tests: sizes unlike any real model's, values that differ where a coincidence (heads ==
kv_heads, key size == value size, all entries rotated, top == experts, one stream, a window that covers everything) would hide a fault, and
weights reshaped so that faults show."""

from __future__ import annotations

import json
from pathlib import Path

import torch


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=6, top=3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def ramp(factor=6.0, original=40, fast=9.0, slow=0.7):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent(heads=3, dim=12, rot_dim=8, vdim=20, kv_rank=24, q_rank=28, size=11, base=90.0, scaling=ramp(), scale=0.5, mlp=None):
    rot = {"dims": rot_dim, "base": base}
    if scaling is not None:
        rot["scaling"] = scaling
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "rot": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale, "mask": {"size": size}}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def gated(heads=4, kv_heads=2, dim=16, vdim=24, rot=12, base=70.0, scale=0.4, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base}, "scale": scale}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def again(layers, j):
    """Layer j once more: the same entry, running with layer j's tensors."""
    return {**layers[j], "weights_of": j}


def model_config(layers, width=52, vocab=127, eps=1e-5, streams=3):
    return {"architecture": "Finolix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams}


# Whole models that differ in every size and option.
_A = [latent(mlp=dense()), gated(mlp=moe()), latent(heads=2, dim=8, rot_dim=4, vdim=9, kv_rank=16, q_rank=12, size=5, base=1e3, mlp=moe(ff=16, experts=3, top=2)),
      gated(heads=6, kv_heads=2, dim=10, vdim=10, rot=10, base=500.0)]
MODEL_A = model_config([*_A, again(_A, 1), again(_A, 0), latent(heads=1, dim=24, rot_dim=2, vdim=16, kv_rank=8, q_rank=40, size=30, mlp=dense(ff=56))])
_B = [gated(heads=3, kv_heads=3, dim=32, vdim=32, rot=6, base=9.0, mlp=moe(ff=8, experts=9, top=4)),
      latent(heads=5, dim=16, rot_dim=12, vdim=8, kv_rank=36, q_rank=20, size=23, base=1e3, scaling=ramp(3.0, 200, 20.0, 1.5), scale=0.3, mlp=dense(ff=72)),
      gated(heads=8, kv_heads=1, dim=48, vdim=40, rot=20, base=1e4, mlp=dense(ff=24))]
MODEL_B = model_config([*_B, again(_B, 1), latent(scaling=None, size=7), again(_B, 0)], width=64, vocab=200, eps=1e-6, streams=2)
# every attention layer has sizes that the tensor-core kernels take in bfloat16, and its only router stands in the last layer, where a choice
# that a rounding step turns over spoils one row and no later one
_C = [latent(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=48, q_rank=64, size=33, base=500.0, scale=0.2, mlp=dense(ff=48)),
      gated(heads=6, kv_heads=2, dim=64, vdim=64, rot=32, base=1e3, scale=0.2, mlp=dense(ff=32)),
      gated(heads=4, kv_heads=4, dim=128, vdim=128, rot=128, base=1e4, scale=0.1)]
MODEL_C = model_config([*_C, again(_C, 0), again(_C, 1), latent(heads=8, dim=64, rot_dim=32, vdim=64, kv_rank=96, q_rank=32, size=50, base=1e4,
                                                              scaling=ramp(16.0, 100, 12.0, 1.0), scale=0.15, mlp=moe(ff=32, experts=5, top=2))],
                       width=72, vocab=150, streams=4)


def make_folder(tmp: Path, config: dict, name: str, seed: int = 0, sharpen: float = 2.0, strength: float = 1.0) -> Path:
    """A model folder with random bfloat16 weights, then reshaped so that faults show: queries and keys are scaled up for peaked attention (a lost,
    doubled or wrongly placed key changes the output), sinks take a visible share, norm weights leave zero, layer scales and the streams' weights
    differ from one another and mix for good, routers' logits and biases are spread out, gates and experts leave their linear stretch.
    ``strength`` < 1 scales all of that down towards plain random weights, for 16-bit runs of deep models, where every factor here also
    multiplies what a rounding step does."""
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
        elif k.endswith((".norm1", ".norm2", "final.norm")):
            f = f * 4
        elif k.endswith((".ls1", ".ls2")):
            f = 0.9 + f * 5
        elif k.endswith((".in", ".out")):
            f = 0.6 + f * 6
        elif k.endswith((".hc1.mix", ".hc2.mix")):
            f = torch.eye(f.shape[0]) * 0.8 + f * 3
        elif k.endswith(".sink"):
            f = 0.5 + f * 20
        elif k.endswith((".uq", ".uk", ".dkv", ".mix.q", ".mix.k")):
            f = f * by(3)
        elif k.endswith(".router"):
            f = f * by(5)
        elif k.endswith(".router.b"):
            f = f * 12
        elif k.endswith((".gate", ".up")) and ".mlp." in k:
            f = f * by(4)
        elif k.endswith(".mix.g"):
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
    from plain import finolix_plain as FP

    key = (str(folder), tuple(ids))
    if key not in _cache:
        if str(folder) not in _cache:
            _cache[str(folder)] = FP.read_model(folder, torch.float64)
        cfg, w = _cache[str(folder)]
        margins: list = []
        _cache[key] = FP.forward(cfg, w, ids, margins=margins).float()
        _cache[("margin",) + key] = torch.stack(margins).min(0).values.float() if margins else torch.full((len(ids),), float("inf"))
    return _cache[key]


def router_margins(folder: Path, ids: list[int]) -> torch.Tensor:
    """Per position, the smallest margin by which any layer's router decided (``inf`` without routers)."""
    plain_logits(folder, ids)
    return _cache[("margin", str(folder), tuple(ids))]

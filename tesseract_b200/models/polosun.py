"""Polosun: latent attention, retention and real-gated recurrence layers, mixer and feed-forward side by side, RMS norms of one
gain and depth averaging. This module reads its ``config.json``; the model itself is ``HybridModel``."""
from __future__ import annotations

import torch

from .hybrid import (HybridConfig, HybridModel, LatentSpec, LayerSpec, RetentionSpec, RGLRUSpec, Rotary, SiluGLUSpec, Yarn)

NAME = "Polosun"


def _rotary(m: dict, dims: int) -> Rotary:
    s = m.get("scaling")
    yarn = Yarn(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None
    return Rotary(dims, float(m["base"]), yarn)


def _mixer(kind: str, m: dict):
    if kind == "latent_attention":
        rot = int(m["rot_dim"])
        return LatentSpec(int(m["heads"]), int(m["dim"]), rot, int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]),
                          _rotary(m["rot"], rot))
    if kind == "retention":
        return RetentionSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(float(d) for d in m["decay"]),
                             _rotary(m["rot"], int(m["rot"]["dims"])))
    if kind == "rglru":
        return RGLRUSpec(int(m["width"]), int(m["blocks"]), int(m["conv"]))
    raise ValueError(f"{NAME}: unknown mixer type {kind!r}")


def _mlp(m):
    if m is None:
        return None
    if m.get("kind") != "dense":
        raise ValueError(f"{NAME}: unknown feed-forward kind {m.get('kind')!r}")
    return SiluGLUSpec(int(m["ff"]))


def config_from_dict(obj: dict, dtype: torch.dtype = torch.bfloat16) -> HybridConfig:
    try:
        layers = [LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in obj["layers"]]
        return HybridConfig(vocab_size=int(obj["vocab"]), width=int(obj["width"]), layers=layers, eps=float(obj["norm"]["eps"]),
                            dtype=dtype, architecture=NAME, form="parallel", residual_mult=float(obj["residual_mult"]),
                            depth_average=True, tied=False)
    except KeyError as e:
        raise ValueError(f"{NAME}: config lacks {e}") from None


def config_to_dict(c: HybridConfig) -> dict:
    def rot(r: Rotary) -> dict:
        out = {"base": r.base, "dims": r.dims}
        if r.scaling is not None:
            s = r.scaling
            out["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
        return out

    def layer(s: LayerSpec) -> dict:
        m = s.mixer
        if isinstance(m, LatentSpec):
            kind, d = "latent_attention", {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                                           "scale": m.scale, "rot": rot(m.rotary)}
        elif isinstance(m, RetentionSpec):
            kind, d = "retention", {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay), "rot": rot(m.rotary)}
        else:
            kind, d = "rglru", {"width": m.width, "blocks": m.blocks, "conv": m.conv}
        return {"type": kind, "mixer": d, "mlp": {"kind": "dense", "ff": s.mlp.ff} if s.mlp is not None else None}
    return {"architecture": NAME, "vocab": c.vocab_size, "width": c.width, "norm": {"eps": c.eps}, "residual_mult": c.residual_mult,
            "layers": [layer(s) for s in c.layers]}


def build(config: HybridConfig, device=None) -> HybridModel:
    return HybridModel(config, device=device)


def layer_cycle(n: int, latent: LatentSpec, ret: RetentionSpec, rec: RGLRUSpec, ff: int) -> list:
    """``n`` layers: retention, latent attention, recurrence, and again."""
    kinds = (ret, latent, rec)
    return [LayerSpec(kinds[i % 3], SiluGLUSpec(ff)) for i in range(n)]


def preset(name: str, dtype: torch.dtype) -> HybridConfig:
    """Random-weight sizes for examples and benchmarks."""
    if name == "tiny":
        W, V, n, ff = 64, 64, 3, 128
        latent = LatentSpec(4, 16, 8, 16, 32, 24 ** -0.5, Rotary(8, 1e4))
        ret = RetentionSpec(4, 16, 32, (0.9, 0.96, 0.98, 0.99), Rotary(16, 1e4))
        rec = RGLRUSpec(96, 4, 4)
    elif name == "small":
        W, V, n, ff = 512, 4096, 6, 1024
        latent = LatentSpec(8, 64, 32, 64, 256, 96 ** -0.5, Rotary(32, 1e4, Yarn(4.0, 4096, 32.0, 1.0)))
        ret = RetentionSpec(4, 128, 128, (0.97, 0.985, 0.993, 0.997), Rotary(128, 1e4))
        rec = RGLRUSpec(512, 4, 4)
    else:
        raise ValueError(f"{NAME}: unknown preset {name!r} (tiny | small)")
    return HybridConfig(V, W, layer_cycle(n, latent, ret, rec, ff), None, 1e-6, 1.0, dtype, architecture=NAME, form="parallel",
                        residual_mult=0.8, depth_average=True, tied=False)

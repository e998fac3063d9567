"""Fozelix: gated-delta and chunked-attention layers with Dynamic Tanh norms around every sublayer, a looped range of layers
and a clamped GLU. This module reads its ``config.json``; the model itself is ``HybridModel``."""
from __future__ import annotations

import torch

from .hybrid import AttentionSpec, DeltaSpec, GLUSpec, HybridConfig, HybridModel, LayerSpec, LoopSpec

NAME = "Fozelix"


def _mixer(kind: str, m: dict):
    if kind == "attention":
        size = int(m["mask"]["size"])
        if size < 1:
            raise ValueError(f"{NAME}: mask.size must be positive")
        return AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), size)
    if kind == "delta":
        return DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
    raise ValueError(f"{NAME}: unknown mixer type {kind!r}")


def _mlp(m):
    if m is None:
        return None
    if m.get("kind") != "dense":
        raise ValueError(f"{NAME}: unknown feed-forward kind {m.get('kind')!r}")
    return GLUSpec(int(m["ff"]), float(m["limit"]))


def config_from_dict(obj: dict, dtype: torch.dtype = torch.bfloat16) -> HybridConfig:
    try:
        layers = [LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in obj["layers"]]
        loop = obj.get("loop")
        return HybridConfig(
            vocab_size=int(obj["vocab"]), width=int(obj["width"]), layers=layers,
            loop=LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None,
            eps=float(obj["norm"]["eps"]), embedding_scale=float(obj["embedding"]["scale"]), dtype=dtype, architecture=NAME)
    except KeyError as e:
        raise ValueError(f"{NAME}: config lacks {e}") from None


def config_to_dict(c: HybridConfig) -> dict:
    def layer(s: LayerSpec) -> dict:
        m = s.mixer
        mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
        if isinstance(m, AttentionSpec):
            mixer.update(scale=m.scale, mask={"size": m.chunk})
        else:
            mixer["conv"] = m.conv
        mlp = {"kind": "dense", "ff": s.mlp.ff, "limit": s.mlp.limit} if s.mlp is not None else None
        return {"type": "attention" if isinstance(m, AttentionSpec) else "delta", "mixer": mixer, "mlp": mlp}
    out = {"architecture": NAME, "vocab": c.vocab_size, "width": c.width, "embedding": {"scale": c.embedding_scale},
           "norm": {"eps": c.eps}, "layers": [layer(s) for s in c.layers]}
    if c.loop is not None:
        out["loop"] = {"start": c.loop.start, "stop": c.loop.stop, "times": c.loop.times}
    return out


def build(config: HybridConfig, device=None) -> HybridModel:
    return HybridModel(config, device=device)


def preset(name: str, dtype: torch.dtype) -> HybridConfig:
    """Random-weight sizes for examples and benchmarks."""
    if name == "tiny":
        W, V, n, ff = 64, 64, 3, 128
        att = AttentionSpec(4, 2, 16, 16, 0.25, 24)
        dlt = DeltaSpec(4, 2, 16, 16, 4)
    elif name == "small":
        W, V, n, ff = 512, 4096, 4, 1024
        att = AttentionSpec(4, 2, 128, 128, 128 ** -0.5, 512)
        dlt = DeltaSpec(4, 2, 128, 128, 4)
    else:
        raise ValueError(f"{NAME}: unknown preset {name!r} (tiny | small)")
    layers = [LayerSpec(att if i % 4 == 3 or i == n - 1 else dlt, GLUSpec(ff, 7.0)) for i in range(n)]
    return HybridConfig(V, W, layers, LoopSpec(1, n, 2), 1e-5, 1.0, dtype, architecture=NAME)

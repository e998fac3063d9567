"""Vobotar: attention with capped scores and values mixed across layers, and layers of windowed attention beside a recurrence (time
mixing or state-space duality); norms on what the sublayers return, and a side input per token. This module reads its
``config.json``; the model itself is ``HybridModel``."""
from __future__ import annotations

import torch

from .hybrid import (HybridConfig, HybridModel, LayerSpec, Rotary, ShapedAttentionSpec, SideBySideSpec, SiluGLUSpec, SSDSpec,
                     TimeMixSpec)

NAME = "Vobotar"
RANK = 32                  # inputs of the decay where neither the weights nor the config say


def _sizes(m: dict) -> tuple:
    return int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"])


def _window(m: dict) -> int:
    size = int(m["mask"]["size"])
    if size < 1:
        raise ValueError(f"{NAME}: mask.size must be positive")
    return size


def _capped(m: dict) -> ShapedAttentionSpec:
    rot = Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"]), neighbours=True)
    return ShapedAttentionSpec(*_sizes(m), norm="head", rotary=rot, softcap=float(m["softcap"]), sink="one", gate="element",
                               v_mix=bool(m.get("v_mix", False)))


def _biased(m: dict) -> ShapedAttentionSpec:
    return ShapedAttentionSpec(*_sizes(m), window=_window(m), bias=True, keys_as_values=True, norm="unit", distance_bias=True,
                               sink="learned", gate="head")


def _rotated(m: dict) -> ShapedAttentionSpec:
    rot = Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"]))
    return ShapedAttentionSpec(*_sizes(m), window=_window(m), bias=True, norm="whole", rotary=rot, gate="head")


def _mixer(kind: str, m: dict, rank):
    if kind == "attention":
        return _capped(m)
    if kind == "parallel":
        r = m["right"]
        left, right = _biased(m["left"]), TimeMixSpec(int(r["heads"]), int(r["dim"]), int(rank or r.get("rank", RANK)))
    elif kind == "parallel_2":
        r = m["right"]
        left = _rotated(m["left"])
        right = SSDSpec(int(r["heads"]), int(r["vdim"]), int(r["state"]), int(r["groups"]), int(r["conv"]), int(r["norm_groups"]))
    else:
        raise ValueError(f"{NAME}: unknown mixer type {kind!r}")
    return SideBySideSpec(left, right, float(m["left_scale"]), float(m["right_scale"]))


def _mlp(m):
    if m is None:
        return None
    if m.get("kind") != "dense":
        raise ValueError(f"{NAME}: unknown feed-forward kind {m.get('kind')!r}")
    return SiluGLUSpec(int(m["ff"]))


def config_from_dict(obj: dict, dtype: torch.dtype = torch.bfloat16, shapes=None) -> HybridConfig:
    """``shapes``: name -> shape of the weights, which say how many inputs the decays have."""
    rank = lambda i: (shapes or {}).get(f"l{i}.mix.right.w1", (0,))[0]   # noqa: E731
    try:
        layers = [LayerSpec(_mixer(l["type"], l["mixer"], rank(i)), _mlp(l.get("mlp"))) for i, l in enumerate(obj["layers"])]
        return HybridConfig(vocab_size=int(obj["vocab"]), width=int(obj["width"]), layers=layers, eps=float(obj["norm"]["eps"]),
                            embedding_scale=float(obj["embedding"]["scale"]), dtype=dtype, architecture=NAME, form="post",
                            token_side=int(obj["token_side"]["dim"]))
    except KeyError as e:
        raise ValueError(f"{NAME}: config lacks {e}") from None


def config_to_dict(c: HybridConfig) -> dict:
    def attention(m: ShapedAttentionSpec) -> dict:
        d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
        if m.rotary is not None:
            d["rot"] = {"base": m.rotary.base, "dims": m.rotary.dims}
        if m.window:
            d["mask"] = {"size": m.window}
        return d

    def layer(s: LayerSpec) -> dict:
        m = s.mixer
        if isinstance(m, ShapedAttentionSpec):
            kind, d = "attention", {**attention(m), "softcap": m.softcap, "v_mix": m.v_mix}
        else:
            r = m.right
            if isinstance(r, TimeMixSpec):
                kind, right = "parallel", {"heads": r.heads, "dim": r.dim, "rank": r.rank}
            else:
                kind, right = "parallel_2", {"heads": r.heads, "vdim": r.vdim, "state": r.state, "groups": r.groups, "conv": r.conv,
                                             "norm_groups": r.norm_parts}
            d = {"left": attention(m.left), "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}
        return {"type": kind, "mixer": d, "mlp": {"kind": "dense", "ff": s.mlp.ff} if s.mlp is not None else None}
    return {"architecture": NAME, "vocab": c.vocab_size, "width": c.width, "norm": {"eps": c.eps}, "embedding": {"scale": c.embedding_scale},
            "token_side": {"dim": c.token_side}, "layers": [layer(s) for s in c.layers]}


def build(config: HybridConfig, device=None) -> HybridModel:
    return HybridModel(config, device=device)


def layer_cycle(n: int, att: ShapedAttentionSpec, mixed: SideBySideSpec, dual: SideBySideSpec, ff: int) -> list:
    """``n`` layers: attention, attention beside time mixing, attention beside state-space duality, and again."""
    kinds = (att, mixed, dual)
    return [LayerSpec(kinds[i % 3], SiluGLUSpec(ff)) for i in range(n)]


def standard_layers(n: int, heads: int, kv_heads: int, dim: int, window: int, mix_heads: int, mix_dim: int, rank: int, dual_heads: int,
                    dual_vdim: int, state: int, ff: int) -> list:
    """A cycle whose three attentions have the same heads."""
    sizes = (heads, kv_heads, dim, dim, dim ** -0.5)
    att = ShapedAttentionSpec(*sizes, norm="head", rotary=Rotary(dim, 1e4, neighbours=True), softcap=30.0, sink="one", gate="element",
                              v_mix=True)
    biased = ShapedAttentionSpec(*sizes, window=window, bias=True, keys_as_values=True, norm="unit", distance_bias=True, sink="learned",
                                 gate="head")
    rotated = ShapedAttentionSpec(*sizes, window=window, bias=True, norm="whole", rotary=Rotary(dim // 2, 1e4), gate="head")
    return layer_cycle(n, att, SideBySideSpec(biased, TimeMixSpec(mix_heads, mix_dim, rank), 0.7, 0.6),
                       SideBySideSpec(rotated, SSDSpec(dual_heads, dual_vdim, state, 1, 4), 0.7, 0.6), ff)


def preset(name: str, dtype: torch.dtype) -> HybridConfig:
    """Random-weight sizes for examples and benchmarks."""
    if name == "tiny":
        W, V, side = 64, 64, 8
        layers = standard_layers(3, 4, 2, 16, 24, 4, 16, 8, 4, 32, 16, 128)
    elif name == "small":
        W, V, side = 512, 4096, 32
        layers = standard_layers(6, 8, 4, 64, 256, 8, 64, 32, 16, 64, 64, 1024)
    else:
        raise ValueError(f"{NAME}: unknown preset {name!r} (tiny | small)")
    return HybridConfig(V, W, layers, eps=1e-6, embedding_scale=W ** 0.5, dtype=dtype, architecture=NAME, form="post", token_side=side)

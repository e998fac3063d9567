"""Tonilix: pre-normed layers of a delta rule whose decays are per key channel, and of attention beside gated linear attention; feed-forwards
are gated by GELU or mixtures of squared-ReLU experts. Positions enter as a sinusoid at the embedding and as queries that grow with them;
a mixer's input is mixed with the one of the token before. This module reads its ``config.json``; the model itself is ``HybridModel``."""
from __future__ import annotations

import torch

from .hybrid import (Choice, DeltaSpec, ExpertSpec, GatedLinearSpec, GeluGLUSpec, HybridConfig, HybridModel, LayerSpec, ShapedAttentionSpec,
                     SideBySideSpec)

NAME = "Tonilix"
RANK = 32                  # inputs of the low-rank products where neither the weights nor the config say


def _attention(m: dict) -> ShapedAttentionSpec:
    t = m["q_temp"]
    return ShapedAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), bias=True, gate="element",
                               q_temp=(float(t["coef"]), float(t["every"])), out_bias=True)


def _mixer(kind: str, m: dict, rank):
    """``rank(name, sizes, key)``: inputs of a low-rank product."""
    if kind == "channel_delta":
        return DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]), rank("a1", m, "decay_rank"),
                         rank("g1", m, "gate_rank"))
    if kind == "parallel":
        r = m["right"]
        right = GatedLinearSpec(int(r["heads"]), int(r["dim"]), int(r["vdim"]), float(r["tau"]), rank("right.a1", r, "rank"))
        return SideBySideSpec(_attention(m["left"]), right, float(m["left_scale"]), float(m["right_scale"]))
    raise ValueError(f"{NAME}: unknown mixer type {kind!r}")


def _mlp(m):
    if m is None:
        return None
    if m.get("kind") == "dense":
        return GeluGLUSpec(int(m["ff"]))
    if m.get("kind") == "moe":
        r = m["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        return ExpertSpec(int(m["expert"]["ff"]), Choice(int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]), float(r["scale"])))
    raise ValueError(f"{NAME}: unknown feed-forward kind {m.get('kind')!r}")


def config_from_dict(obj: dict, dtype: torch.dtype = torch.bfloat16, shapes=None) -> HybridConfig:
    """``shapes``: name -> shape of the weights, which say how many inputs the low-rank products have."""
    def rank(i):
        return lambda name, sizes, key: int((shapes or {}).get(f"l{i}.mix.{name}", (sizes.get(key, RANK),))[0])
    try:
        layers = [LayerSpec(_mixer(l["type"], l["mixer"], rank(i)), _mlp(l.get("mlp"))) for i, l in enumerate(obj["layers"])]
        return HybridConfig(vocab_size=int(obj["vocab"]), width=int(obj["width"]), layers=layers, eps=float(obj["norm"]["eps"]), dtype=dtype,
                            architecture=NAME, form="pre", tied=False, norm_parts=int(obj["norm"]["groups"]), layer_scale=True, token_shift=True,
                            sinusoid=True, embed_norm=True)
    except KeyError as e:
        raise ValueError(f"{NAME}: config lacks {e}") from None


def config_to_dict(c: HybridConfig) -> dict:
    def mixer(m):
        if isinstance(m, DeltaSpec):
            return "channel_delta", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv,
                                     "decay_rank": m.decay_rank, "gate_rank": m.gate_rank}
        a, r = m.left, m.right
        left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                "q_temp": {"coef": a.q_temp[0], "every": a.q_temp[1]}}
        right = {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "tau": r.tau, "rank": r.rank}
        return "parallel", {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}

    def mlp(m):
        if m is None:
            return None
        if isinstance(m, GeluGLUSpec):
            return {"kind": "dense", "ff": m.ff}
        r = m.choice
        return {"kind": "moe", "expert": {"ff": m.ff}, "router": {"experts": r.experts, "top": r.top, "scale": r.scale,
                                                                  "groups": {"count": r.groups, "keep": r.keep}}}

    def layer(s: LayerSpec) -> dict:
        kind, d = mixer(s.mixer)
        return {"type": kind, "mixer": d, "mlp": mlp(s.mlp)}
    return {"architecture": NAME, "vocab": c.vocab_size, "width": c.width, "norm": {"eps": c.eps, "groups": c.norm_parts},
            "layers": [layer(s) for s in c.layers]}


def build(config: HybridConfig, device=None) -> HybridModel:
    return HybridModel(config, device=device)


def layer_cycle(n: int, delta: DeltaSpec, pair: SideBySideSpec, dense: GeluGLUSpec, experts: ExpertSpec) -> list:
    """``n`` layers: two of the delta rule to every one of attention beside gated linear attention; the first feed-forward is dense."""
    return [LayerSpec(pair if i % 3 == 2 else delta, experts if i else dense) for i in range(n)]


def standard_layers(n: int, heads: int, kv_heads: int, dim: int, delta_heads: int, delta_dim: int, rank: int, linear_heads: int, linear_dim: int,
                    ff: int, expert_ff: int, choice: Choice) -> list:
    att = ShapedAttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, bias=True, gate="element", q_temp=(0.1, 2048.0), out_bias=True)
    pair = SideBySideSpec(att, GatedLinearSpec(linear_heads, linear_dim, linear_dim, 16.0, rank), 0.7, 0.6)
    delta = DeltaSpec(delta_heads, delta_heads, delta_dim, delta_dim, 4, rank, rank)
    return layer_cycle(n, delta, pair, GeluGLUSpec(ff), ExpertSpec(expert_ff, choice))


def preset(name: str, dtype: torch.dtype) -> HybridConfig:
    """Random-weight sizes for examples and benchmarks."""
    if name == "tiny":
        W, V = 64, 64
        layers = standard_layers(3, 4, 2, 16, 4, 16, 8, 4, 16, 128, 32, Choice(8, 2, 4, 2, 1.0))
    elif name == "small":
        W, V = 512, 4096
        layers = standard_layers(6, 8, 4, 64, 8, 64, 32, 8, 64, 1024, 256, Choice(32, 4, 4, 2, 2.0))
    else:
        raise ValueError(f"{NAME}: unknown preset {name!r} (tiny | small)")
    return HybridConfig(V, W, layers, eps=1e-6, dtype=dtype, architecture=NAME, form="pre", tied=False, norm_parts=4, layer_scale=True,
                        token_shift=True, sinusoid=True, embed_norm=True)

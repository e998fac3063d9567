"""Vobotar (attention with chosen parts, time mixing, state-space duality, post-normed layers, a side input per token) against the
plain statements of ``vobotar_oracle``: every mechanism alone, prompts, portions, batches, decoding, reuse of pages and slots, and
generation through the framework's entry points. The same tests run on the CPU and, marked ``gpu``, on the kernels."""
import io
import json
import math

import numpy as np
import pytest
import torch

import vobotar_oracle as oracle
from tesseract_b200 import ops
from tesseract_b200.models import GenerateConfig, load_pretrained, vobotar
from tesseract_b200.models.hybrid import (GLUSpec, HybridConfig, HybridModel, LayerSpec, ShapedAttentionSpec, SideBySideSpec, SiluGLUSpec,
                                          SSDSpec, TimeMixSpec)
from tesseract_b200.models.registry import resolve
from tesseract_b200.models.scheduler import ContinuousBatchingScheduler, EngineConfig
from tesseract_b200.nn.hybrid import SSD, ShapedAttention, TimeMix
from tesseract_b200.nn.ragged import HybridCache, HybridSequence, RaggedBatch
from tesseract_b200.ops.masks import Window
from tesseract_b200.ops.ragged import AttentionGeometry, ScoreForm
from tesseract_b200.ops.rotary import Rotary, rotate_stored
from tesseract_b200.ops.ssd import SSDGeometry, part_norm_
from tesseract_b200.ops.timemix import TimeMixGeometry, token_shift
from tesseract_b200.serving import HybridEngine, make_engine

KINDS = [("cpu", "float32"), ("cpu", "bfloat16"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu),
         pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]
# relative error of a row of logits: bf16 rounding alone reaches 0.13 in single rows; a mechanism that is off by one
# token or factor shows as 0.3 and more
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.2}
MEAN_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.03}


def mlp(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def att(heads, kv, dim, vdim, dims, softcap, mix=True, scale=0.3, base=1e3, ff=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims},
                                           "scale": scale, "softcap": softcap, "v_mix": mix}, "mlp": mlp(ff)}


def par(heads, kv, dim, window, mix_heads, mix_dim, rank, scale=0.4, scales=(0.9, 0.6), ff=None):
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "mask": {"size": window}, "scale": scale},
                                          "right": {"heads": mix_heads, "dim": mix_dim, "rank": rank}, "left_scale": scales[0],
                                          "right_scale": scales[1]}, "mlp": mlp(ff)}


def par2(heads, kv, dim, vdim, window, dims, ssd_heads, ssd_vdim, state, groups, conv, parts, scale=0.3, base=2e3, scales=(1.3, 0.7), ff=None):
    return {"type": "parallel_2", "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window},
                                                     "rot": {"base": base, "dims": dims}, "scale": scale},
                                            "right": {"heads": ssd_heads, "vdim": ssd_vdim, "state": state, "groups": groups, "conv": conv,
                                                      "norm_groups": parts}, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp(ff)}


def conf(vocab, width, side, layers, eps=1e-5, scale=1.7):
    return {"architecture": "Vobotar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "token_side": {"dim": side}, "layers": layers}


CONFIGS = {
    # sizes that are multiples of nothing, layers without a feed-forward, one that mixes no values between two that do, parts of a norm
    # that cut heads, a window of one token
    "odd": conf(53, 42, 5, [att(6, 3, 10, 7, 6, 4.0, ff=30), par(4, 2, 12, 5, 3, 11, 5, ff=27), par2(3, 1, 9, 14, 7, 4, 6, 10, 7, 3, 3, 4, ff=33),
                            att(4, 2, 8, 9, 8, 2.0, mix=False), att(6, 3, 6, 7, 2, 6.0, ff=21), par2(4, 4, 6, 5, 1, 0, 2, 9, 12, 1, 1, 1),
                            par(5, 5, 7, 9, 2, 8, 20)], 0.5),
    # sizes that the tensor-core kernels take
    "plain": conf(130, 96, 24, [par(4, 2, 64, 40, 3, 32, 16, 0.12, ff=72), att(4, 2, 64, 32, 32, 20.0, scale=0.1, ff=80),
                                par2(8, 2, 48, 64, 70, 16, 4, 32, 64, 2, 4, 2, 0.15, ff=64), att(2, 2, 32, 32, 32, 9.0, ff=48)], 1e-6),
    # heads of 128 and heads, states and sections too large for the fast kernels
    "wide": conf(64, 128, 33, [par(2, 1, 128, 33, 2, 128, 40, 0.08, ff=96), att(3, 1, 100, 128, 60, 12.0, scale=0.1), att(3, 1, 150, 128, 10, 12.0,
                               scale=0.08), par2(9, 1, 128, 70, 20, 128, 2, 136, 128, 1, 4, 1, 0.08), par(1, 1, 200, 17, 1, 150, 70, 0.07),
                               par2(2, 2, 160, 16, 30, 100, 3, 40, 200, 3, 5, 12, 0.08, ff=64)]),
    # one kind each
    "attention": conf(33, 32, 3, [att(4, 1, 16, 8, 12, 3.0, ff=24), att(2, 1, 24, 8, 24, 5.0)], 0.05, 1.0),
    "mixing": conf(40, 48, 8, [par(2, 2, 16, 6, 3, 16, 4, ff=24), par(4, 1, 8, 11, 2, 24, 9)], 1e-4),
    "dual": conf(40, 48, 8, [par2(2, 1, 16, 8, 6, 8, 4, 16, 16, 2, 4, 4, ff=24), par2(4, 2, 8, 8, 13, 8, 2, 32, 24, 1, 2, 1)], 1e-4),
}


def make_weights(config, seed=0):
    """bf16 tensors for every name the model has, sized so that no mechanism fades."""
    g = torch.Generator().manual_seed(seed)
    model = HybridModel(vobotar.config_from_dict(config))

    def draw(name, shape):
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last == "vmix":
            return 0.3 + 0.4 * torch.rand((), generator=g)
        if ".mu." in name:
            return 0.2 + 0.6 * torch.rand(shape, generator=g)
        if last == "w0":
            return 1.5 * r - 2.5
        if last in ("A_log", "dt_bias"):
            return 0.7 * r - 1.5
        if last == "conv":
            return 0.6 * r
        if last in ("u", "D"):
            return 0.6 * r
        if last == "b":
            return 0.4 * r
        if last == "sink":
            return 1.0 + r
        if last == "norm" or last.startswith("norm"):
            return 0.3 * r + (0.0 if name.split(".")[1] in ("norm1", "norm2") or name == "final.norm" else 1.0)
        if name in ("embed", "side.embed"):
            return 0.7 * r
        return r * (1.5 / math.sqrt(shape[-1]))
    w = {n: draw(n, s) for n, s in model.logical_shapes().items()}
    for n in list(w):
        if n.endswith("right.r"):      # the read-out over its own size has the sign of r . k: keep that away from zero
            w[n] = 0.8 * w[n[:-1] + "k"] + 0.6 * w[n]
    return {n: t.to(torch.bfloat16) for n, t in w.items()}


def make_model(config, weights, kind):
    m = HybridModel(vobotar.config_from_dict(config, getattr(torch, kind[1])), device=kind[0])
    assert m.load_tensors(weights) == []
    return m


def tokens_for(config, n, seed=1):
    return np.random.default_rng(seed).integers(0, config["vocab"], n).tolist()


def row_error(got, want):
    got, want = got.double().cpu(), want.double()
    return ((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-6))


def check(got, want, kind, what=""):
    e = row_error(got, want)
    dt = getattr(torch, kind[1])
    assert float(e.max()) < TOL[dt], f"{what}: worst row {int(e.argmax())} of {len(e)}: {float(e.max()):.2e} (limit {TOL[dt]})"
    if len(e) >= 16:
        assert float(e.mean()) < MEAN_TOL[dt], f"{what}: mean {float(e.mean()):.2e}"


_reference, _weights = {}, {}


def reference(name, toks):
    key = (name, tuple(toks))
    if key not in _reference:
        _reference[key] = oracle.run_model(CONFIGS[name], weights_of(name), toks)
    return _reference[key]


def weights_of(name):
    if name not in _weights:
        _weights[name] = make_weights(CONFIGS[name], seed=len(name))
    return _weights[name]


def engine_for(name, kind, blocks=64, block=8, batch=4, **kw):
    m = make_model(CONFIGS[name], weights_of(name), kind)
    return HybridEngine(m, EngineConfig(block_size=block, num_blocks=blocks, max_seq_len=blocks * block, max_batch_size=batch), **kw)


def feed(eng, seq, toks, cuts):
    """Runs ``toks`` through one sequence in portions; logits of every token."""
    out, at = [], 0
    for n in cuts:
        out.append(eng.execute([(seq, toks[at:at + n])], [list(range(n))]))
        at += n
    assert at == len(toks)
    return torch.cat([o.float().cpu() for o in out])


# ---------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dims,dim", [(64, 64), (12, 19), (2, 5), (0, 8)])
def test_neighbour_rotation_layout_and_far_positions(dims, dim):
    r = Rotary(dims, 700.0, neighbours=True)
    rot = {"dims": dims, "base": 700.0}
    cols = r.columns(dim).tolist()
    assert len(set(cols)) == dim and max(cols, default=0) < r.stored(dim)
    for i in range(dims // 2):
        assert cols[2 * i + 1] - cols[2 * i] == r.hp
    table = r.table(9000)
    x = torch.randn(3, 2, dim, dtype=torch.float64)
    stored = torch.zeros(3, 2, r.stored(dim))
    stored[..., cols] = x.float()
    got = rotate_stored(stored, table, torch.tensor([5, 0, 8999]))[..., cols]
    assert (got - oracle.rotate_pairs(x, [5, 0, 8999], rot)).abs().max() < 1e-5


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("W,cols", [(40, 48), (37, 48), (256, 256), (1030, 1040), (2304, 2304), (9000, 9008)])
def test_post_norm_step_in_every_form(kind, W, cols):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(W)
    T, V, eps = 7, 19, 1e-2
    rnd = lambda *s: torch.randn(*s, generator=g)   # noqa: E731
    table = torch.zeros(V, cols, dtype=dt)
    table[:, :W] = rnd(V, W)
    toks = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    form = dict(out_cols=cols, out_dtype=dt)
    htol = 3e-5 if dt == torch.float32 else 0.04
    x = torch.empty(T, W, device=dev)
    h = ops.post_norm_step(x, tokens=toks.to(dev), table=table.to(dev), scale=2.5, **form)
    want = table[toks.long(), :W].double() * 2.5
    assert (x.cpu().double() - want).abs().max() < 1e-6 and (h[:, :W].cpu().double() - want).abs().max() < htol
    assert float(h[:, W:].abs().sum()) == 0.0
    y, gain, final = (0.1 * rnd(T, cols)).to(dt), 1 + 0.3 * rnd(W), 1 + 0.3 * rnd(W)
    for last in (False, True):
        x0 = rnd(T, W)
        x = x0.clone().to(dev)
        h = ops.post_norm_step(x, y.to(dev), gain.to(dev), eps, final=final.to(dev) if last else None, **form)
        want = x0.double() + oracle.over_rms(y[:, :W].double(), eps) * gain.double()
        assert (x.cpu().double() - want).abs().max() < 2e-5               # the residual stays in 32-bit whatever the type
        if last:
            want = oracle.over_rms(want, eps) * final.double()
        assert (h[:, :W].cpu().double() - want).abs().max() < htol * max(1.0, float(want.abs().max()) / 4)
        assert float(h[:, W:].abs().sum()) == 0.0


@pytest.mark.parametrize("kind", KINDS)
def test_side_input_looks_up_its_layers_columns(kind):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(0)
    V, L, dim = 11, 3, 21
    table = torch.randn(V, L * dim, generator=g).to(dt)
    toks = torch.tensor([3, 10, 0, 3], dtype=torch.int32)
    z = torch.zeros(4, 32, dtype=dt)
    z[:, :dim] = (3 * torch.randn(4, dim, generator=g)).to(dt)
    for layer in range(L):
        got = ops.gelu_lookup(z.to(dev), toks.to(dev), table.to(dev), layer * dim, dim).cpu().double()
        want = oracle.gelu_tanh(z[:, :dim].double()) * table[toks.long(), layer * dim:(layer + 1) * dim].double()
        assert (got[:, :dim] - want).abs().max() < (1e-5 if dt == torch.float32 else 0.06) and float(got[:, dim:].abs().sum()) == 0.0


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("M,starts,N,K", [(3, (0, 128), 150, 48), (70, (0, 128, 384, 512), 600, 112), (200, (0, 256, 512), 768, 192),
                                          (300, (0, 128, 256, 384, 512, 640), 650, 80), (5, (0, 256, 1024, 1280), 1296, 2048)])
def test_one_product_of_several_inputs(kind, M, starts, N, K):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(M)
    xs = torch.randn(len(starts), M, K, generator=g).to(dt)
    w = (torch.randn(N, K, generator=g) * K ** -0.5).to(dt)
    got = ops.project_inputs(xs.to(dev), w.to(dev), starts).cpu().double()
    for i, (a, b) in enumerate(zip(starts, list(starts[1:]) + [N])):
        want = xs[i].double() @ w[a:b].double().t()
        assert (got[:, a:b] - want).abs().max() < (2e-4 if dt == torch.float32 else 0.03), i
    with pytest.raises(ValueError, match="starts"):
        ops.project_inputs(xs.to(dev), w.to(dev), tuple(s + 8 * (i == 1) for i, s in enumerate(starts)))


def packed(block, T, values, kind):
    """The block's packed projection rows with the given logical values."""
    p = torch.zeros(T, block.cols)
    for name, rows in block._rows().items():
        p[:, rows] = values[name].reshape(T, -1).float()
    return p.to(getattr(torch, kind[1])).to(kind[0])


def run_core(block, proj, cuts, kind, block_size=8, first_values=None):
    """Feeds rows of ``proj`` through a cache of one sequence whose slot and pages hold what an earlier one left. ``first_values``
    [T, heads, D]: what the first layer that mixes values holds."""
    T = proj.shape[0]
    n = (T + block_size - 1) // block_size
    spec = block.run_spec()
    runs = [spec, spec] if first_values is not None else [spec]
    cache = HybridCache(runs, n + 3, block_size, 2, (n + 3) * block_size, block.dtype, kind[0])
    run = cache.runs[-1]
    for t in run[:2]:
        t.copy_(torch.randn(t.shape).to(t.dtype))
    cache.allocator.allocate()                   # the sequence's pages and slot are not the pool's first
    cache.slot_allocator.allocate()
    seq, got, at = HybridSequence(cache), [], 0
    for n in cuts:
        b = RaggedBatch(cache, [(seq, [0] * n)], None, list(block.masks), 0, list(block.tiles))
        if first_values is not None:
            sl = b.slots.long()
            cache.runs[0][1][sl // block_size, :, sl % block_size] = first_values[at:at + n].to(kind[0], block.dtype)
        got.append(block.core(proj[at:at + n].contiguous(), run, b).float().cpu())
        b.commit()
        at += n
    assert at == T
    return torch.cat(got).double(), run, seq


ATT = {
    "capped": dict(heads=4, kv=2, dim=12, vdim=20, norm="head", rotary=Rotary(8, 90.0, neighbours=True), softcap=2.0, sink="one", gate="element"),
    "capped64": dict(heads=6, kv=3, dim=64, vdim=40, norm="head", rotary=Rotary(64, 90.0, neighbours=True), softcap=8.0, sink="one",
                     gate="element"),
    "mixed": dict(heads=3, kv=3, dim=128, vdim=64, norm="head", rotary=Rotary(6, 90.0, neighbours=True), softcap=9.0, sink="one", gate="element",
                  v_mix=True),
    "biased": dict(heads=6, kv=2, dim=14, vdim=14, window=9, bias=True, keys_as_values=True, norm="unit", slopes=True, sink="learned",
                   gate="head"),
    "biased64": dict(heads=8, kv=1, dim=64, vdim=64, window=50, bias=True, keys_as_values=True, norm="unit", slopes=True, sink="learned",
                     gate="head"),
    "biased128": dict(heads=9, kv=1, dim=100, vdim=100, window=128, bias=True, keys_as_values=True, norm="unit", slopes=True, sink="learned",
                      gate="head"),
    "whole": dict(heads=5, kv=1, dim=9, vdim=22, window=1, bias=True, norm="whole", rotary=Rotary(4, 90.0), gate="head"),
    "whole64": dict(heads=4, kv=4, dim=50, vdim=64, window=129, bias=True, norm="whole", rotary=Rotary(20, 90.0), gate="head"),
    "long": dict(heads=2, kv=1, dim=200, vdim=130, window=40, bias=True, norm="whole", rotary=Rotary(100, 90.0), gate="head"),
    # parts that the design does not put together, a cap that bounds nothing
    "loose": dict(heads=2, kv=1, dim=64, vdim=48, window=140, norm="head", slopes=True, softcap=90.0, sink="learned", gate="head"),
    "bare": dict(heads=2, kv=1, dim=64, vdim=64),
    "sinks": dict(heads=2, kv=2, dim=64, vdim=64, sink="learned", norm="unit", slopes=True, softcap=3.0, window=77, gate="element"),
}


def make_attention(name, kind, scale, seed=0):
    a, dt = ATT[name], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(seed)
    slopes = torch.tensor(oracle.distance_slopes(a["heads"])).float() if a.get("slopes") else None
    form = ScoreForm(scale, Window(a["window"]) if "window" in a else 0, a.get("softcap", 0.0), slopes,
                     torch.zeros(a["heads"]) if a.get("sink") == "one" else None)
    blk = ShapedAttention(32, a["heads"], a["kv"], a["dim"], a["vdim"], form, 1e-2, dt, kind[0], a.get("bias", False),
                          a.get("keys_as_values", False), a.get("norm", ""), a.get("rotary"), a.get("sink") == "learned", a.get("v_mix", False),
                          a.get("gate", ""))
    w = {}
    for n, s in blk.logical_shapes().items():
        w[n] = (torch.zeros(s) if len(s) == 2 else torch.tensor(0.3) if n == "vmix" else 1.0 + 0.4 * torch.randn(s, generator=g) if "norm" in n
                else torch.randn(s, generator=g)).to(torch.bfloat16)
    blk.load(w)
    return blk, {n: t.double() for n, t in w.items()}


def attention_of(name, blk, w, val, scale, out_scale, dt, first=None):
    a, T = ATT[name], val["q"].shape[0]
    H, G, D, E, eps = a["heads"], a["kv"], a["dim"], a["vdim"], 1e-2
    z = {n: t.to(dt).double() for n, t in val.items()}
    biased = lambda n: z[n] + w[n + ".b"] if a.get("bias") else z[n]   # noqa: E731
    q, k = biased("q"), biased("k")
    v = (k if a.get("keys_as_values") else biased("v")).view(T, G, E)
    if a.get("norm") == "whole":
        q, k = oracle.over_rms(q, eps) * w["q.norm"], oracle.over_rms(k, eps) * w["k.norm"]
    q, k = q.view(T, H, D), k.view(T, G, D)
    if a.get("norm") in ("unit", "head"):
        q, k = oracle.over_rms(q, eps), oracle.over_rms(k, eps)
    if a.get("norm") == "head":
        q, k = q * w["q.norm"], k * w["k.norm"]
    r = a.get("rotary")
    if r is not None:
        turn = oracle.rotate_pairs if r.neighbours else oracle.rotate
        q, k = (turn(t, range(T), {"dims": r.dims, "base": r.base}) for t in (q, k))
    if first is not None:
        v = (1.0 - w["vmix"]) * v + w["vmix"] * first.to(dt).double()
    o = oracle.attend(q, k, v, scale, a.get("window"), a.get("softcap"), oracle.distance_slopes(H) if a.get("slopes") else None,
                      w.get("sink"), a.get("sink") == "one")
    if a.get("gate") == "head":
        o = o * oracle.sigmoid(z["g"])[:, :, None]
    o = o.reshape(T, H * E)
    if a.get("gate") == "element":
        o = o * oracle.sigmoid(z["g"])
    return o * out_scale


def prompt_cuts(T, *edges):
    """Whole, token by token, pairs, and portions that end around the edges."""
    out = [[T], [1] * T, [2] * (T // 2) + [1] * (T % 2)]
    for e in edges:
        if 2 < e < T - 2:
            out += [[e, T - e], [e - 1, 2, T - e - 1], [e + 1] + [1] * min(7, T - e - 1) + ([T - e - 1 - min(7, T - e - 1)] if T - e - 8 > 0 else [])]
    return out


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", list(ATT))
def test_attention_alone(kind, name):
    a, dt = ATT[name], getattr(torch, kind[1])
    T, scale = 150, 1.5 * ATT[name]["dim"] ** -0.5
    blk, w = make_attention(name, kind, scale, seed=len(name))
    blk.out_scale = 0.7
    g = torch.Generator().manual_seed(3)
    val = {n: torch.randn(T, len(r), generator=g) * (0.3 if n in "qk" else 1.0) for n, r in blk._rows().items()}   # (near eps: where it goes shows)
    first = torch.randn(T, a["kv"], a["vdim"], generator=g) if a.get("v_mix") else None
    pool_first = torch.zeros(T, a["kv"], blk.geo.D) if first is not None else None
    if first is not None:
        pool_first[..., :a["vdim"]] = first
    proj = packed(blk, T, val, kind)
    want = attention_of(name, blk, w, val, scale, 0.7, dt, first)
    cols = blk._out_columns()
    cuts = prompt_cuts(T, a.get("window", 64), 128)
    for c in cuts if kind[0] == "cuda" else cuts[:1] + cuts[3:5]:
        got, _, _ = run_core(blk, proj, c, kind, first_values=pool_first)
        err = (got[:, cols] - want).abs().max(1).values
        assert float(err.max()) < (1e-4 if dt == torch.float32 else 0.03), (c[:4], int(err.argmax()))
        rest = [i for i in range(got.shape[1]) if i not in set(cols.tolist())]
        assert float(got[:, rest].abs().sum()) == 0.0
    if a.get("v_mix"):                           # the first such layer keeps its own values
        got, _, _ = run_core(blk, proj, [T], kind)
        assert (got[:, cols] - attention_of(name, blk, w, val, scale, 0.7, dt)).abs().max() < (1e-4 if dt == torch.float32 else 0.03)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name,window", [("whole64", 129), ("biased", 9), ("biased128", 128), ("whole", 1), ("long", 40), ("bare", 10 ** 6), ("capped64", 10 ** 6)])
def test_one_standing_out_key_everywhere(kind, name, window):
    """One key is made to win wherever it is seen and its value to be unmistakable: the queries inside its window return that value,
    those just before and just past it do not -- in prompts, portions and decoding, around page, tile and window edges."""
    a, dt = ATT[name], getattr(torch, kind[1])
    T, H, G, D, E = 290 if kind[0] == "cuda" and name != "capped64" else 150, a["heads"], a["kv"], a["dim"], a["vdim"]
    scale = 8.0 / D if a.get("norm") in ("unit", "head") else 6.0
    blk, w = make_attention(name, kind, scale)
    for n in ("q.b", "k.b", "v.b", "sink"):      # (a loud sink or bias would only make the edges harder to see)
        if n in w:
            w[n] = 0.0 * w[n]
    blk.load({n: t.to(torch.bfloat16) for n, t in w.items()})
    g = torch.Generator().manual_seed(7)
    r = a.get("rotary")
    still = D - 1 if r is None or r.dims < D else None       # a coordinate that does not turn
    for hot in (0, 7, 8, 63, 127, 128, T - 1):
        if hot >= T:
            continue
        val = {n: 0.05 * torch.randn(T, len(rows), generator=g) for n, rows in blk._rows().items()}
        q, k = val["q"].view(T, H, D), val["k"].view(T, G, D)
        if still is not None:
            q[:, :, still], k[hot, :, still] = 5.0, 40.0
        else:
            q[:, :, 0], k[hot, :, 0] = 5.0, 40.0
        if "v" in val:
            val["v"][hot] = 3.0
        if "g" in val:
            val["g"][:] = 20.0
        proj = packed(blk, T, val, kind)
        want = attention_of(name, blk, w, val, scale, 1.0, dt)
        top = float(want.abs().max())
        last = min(T, hot + window)
        if still is not None and not a.get("slopes"):
            assert float(want[hot:last].abs().max(1).values.min()) > 0.5 * top
        if last < T:
            assert float(want[last:].abs().max()) < 0.3 * top
        assert hot == 0 or float(want[:hot].abs().max()) < 0.3 * top
        edge = min(hot + min(window, T), T - 1)
        forms = [[T], [max(hot, 1), 2, T - max(hot, 1) - 2], [hot + 1] + [1] * min(9, T - hot - 1) + [T - hot - 1 - min(9, T - hot - 1)],
                 [max(edge - 3, 1)] + [1] * min(6, T - max(edge - 3, 1)) + [T - max(edge - 3, 1) - min(6, T - max(edge - 3, 1))],
                 [max(edge - 1, 1), 2, T - max(edge - 1, 1) - 2]]
        for c in forms if kind[0] == "cuda" else forms[:4:3]:
            c = [n for n in c if n > 0]
            if sum(c) != T:
                continue
            got, _, _ = run_core(blk, proj, c, kind, block_size=16)
            err = (got[:, blk._out_columns()] - want).abs().max(1).values
            assert float(err.max()) < (2e-4 if dt == torch.float32 else 0.03) * max(top, 1.0), (hot, c[:3], int(err.argmax()))


@pytest.mark.parametrize("kind", KINDS)
def test_a_loud_and_a_silent_sink(kind):
    """A sink far above every score takes all the weight, one far below takes none, whatever the number of keys."""
    dt = getattr(torch, kind[1])
    for name in ("biased", "biased64", "sinks"):
        blk, w = make_attention(name, kind, 0.2)
        T, H = 140, ATT[name]["heads"]
        w["sink"] = torch.where(torch.arange(H) % 2 == 0, 300.0, -300.0).double()
        blk.load({n: t.to(torch.bfloat16) for n, t in w.items()})
        g = torch.Generator().manual_seed(1)
        val = {n: torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
        want = attention_of(name, blk, w, val, 0.2, 1.0, dt)
        assert float(want.view(T, H, -1)[:, ::2].abs().max()) < 1e-50 and float(want.view(T, H, -1)[:, 1::2].abs().max()) > 0.3
        for c in ([T], [100] + [1] * 40):
            got, _, _ = run_core(blk, packed(blk, T, val, kind), c, kind)
            assert (got[:, blk._out_columns()] - want).abs().max() < (1e-4 if dt == torch.float32 else 0.03), (name, len(c))


@pytest.mark.parametrize("kind", KINDS)
def test_token_shift_across_portions_and_slots(kind):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(5)
    W, cols = 37, 48
    blk = TimeMix(W, 2, 8, 4, 1e-5, dt, dev)
    mu = torch.zeros(5, cols)
    mu[:, :W] = torch.rand(5, W, generator=g)
    cache = HybridCache([blk.run_spec()], 40, 8, 3, 96, dt, dev)
    last = cache.runs[0][0]
    last.copy_(torch.randn(last.shape).to(dt))
    rows = {s: torch.zeros(n, cols, dtype=dt) for s, n in (("a", 21), ("b", 13))}
    for t in rows.values():
        t[:, :W] = torch.randn(t.shape[0], W, generator=g).to(dt)
    want = {s: torch.stack([oracle.shifted_mix(t.double(), mu[i].double()) for i in range(5)]) for s, t in rows.items()}
    seqs, at = {s: HybridSequence(cache) for s in rows}, dict.fromkeys(rows, 0)
    for step in ({"a": 1}, {"b": 5, "a": 3}, {"a": 1, "b": 1}, {"b": 2, "a": 9}, {"a": 2}, {"b": 5, "a": 5}):
        b = RaggedBatch(cache, [(seqs[s], [0] * n) for s, n in step.items()])
        h = torch.zeros(b.rows, cols, dtype=dt)
        for i, (s, n) in enumerate(step.items()):
            h[b.row_of[i]:b.row_of[i] + n] = rows[s][at[s]:at[s] + n]
        xs = token_shift(h.to(dev), mu.to(dev), last, b, keep=True).cpu()
        b.commit()
        assert torch.equal(xs[0], h)
        for i, (s, n) in enumerate(step.items()):
            got = xs[1:, b.row_of[i]:b.row_of[i] + n].double()
            assert (got - want[s][:, at[s]:at[s] + n]).abs().max() < (1e-6 if dt == torch.float32 else 0.02), (s, at[s])
            at[s] += n
            assert torch.equal(last[seqs[s].slot, 0].cpu(), rows[s][at[s] - 1])


MIX_SIZES = [(3, 11, 5), (2, 16, 16), (1, 48, 20), (2, 64, 64), (2, 128, 32), (1, 150, 90)]


def mix_case(blk, T, kind, seed, spread=1.0):
    """(proj, oracle's r, k, v, gate, decay, u, weights)"""
    dt, g = getattr(torch, kind[1]), torch.Generator().manual_seed(seed)
    H, D, R = blk.geo.heads, blk.geo.dim, blk.geo.rank
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    w.update(w2=torch.randn(H * D, R, generator=g) * R ** -0.5, w0=spread * torch.randn(H * D, generator=g) - 2.0, u=torch.randn(H, D, generator=g),
             norm=1 + 0.3 * torch.randn(H * D, generator=g))
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    d = {n: t.double() for n, t in w.items()}
    val = {n: torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
    val["k"], val["r"] = 0.5 * val["k"], 0.5 * val["k"] + 0.3 * val["r"]        # (r . k away from zero)
    z = {n: v.to(dt).double() for n, v in val.items()}
    low = torch.tanh(z["w1"]).to(dt).double()
    decay = torch.exp(-torch.exp(low @ d["w2"].t() + d["w0"])).view(T, H, D)
    return packed(blk, T, val, kind), z, decay, d


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,D,R", MIX_SIZES)
@pytest.mark.parametrize("spread", [1.0, 4.0])
def test_time_mixing_alone(kind, H, D, R, spread):
    """Prompts, portions and single tokens against the token-by-token statement; with the wide spread, decays run from nearly 1 to
    exactly 0. The slot had been used before; the state stays in 32-bit."""
    dt = getattr(torch, kind[1])
    T, eps = 141, 1e-2
    blk = TimeMix(32, H, D, R, eps, dt, kind[0])
    blk.out_scale = 0.8
    proj, z, decay, d = mix_case(blk, T, kind, D, spread)
    o, S = oracle.bonus_recurrence(z["r"].view(T, H, D), z["k"].view(T, H, D), z["v"].view(T, H, D), decay, d["u"])
    want = 0.8 * oracle.over_rms(o, eps).reshape(T, H * D) * d["norm"] * oracle.silu(z["g"])
    cols = blk._out_columns()
    tol = 3e-4 if dt == torch.float32 else 0.03
    every = [[T], [64, 1, 63, 13], [1, 2, 15, 1, 16, 17, 89], [2] * 70 + [1], [128] + [1] * 13, [1] * T]
    for cuts in every[:3] if kind[0] == "cpu" else every:
        got, run, seq = run_core(blk, proj, cuts, kind)
        err = (got[:, cols] - want).abs().max(1).values
        assert float(err.max()) < tol * float(want.abs().max()), (cuts[:4], int(err.argmax()))
        state = run[1][seq.slot].cpu().double()[:, :D, :D].transpose(1, 2)
        assert (state - S).abs().max() < (1e-4 if dt == torch.float32 else 1e-3) * float(S.abs().max()), cuts[:4]


@pytest.mark.parametrize("kind", KINDS)
def test_time_mixing_keeps_a_far_token(kind):
    """Everything is silent but one token far back: its trace comes out at the size its channel's decay leaves, across chunks,
    blocks and portions."""
    dt = getattr(torch, kind[1])
    T, H, D = 150, 2, 16
    blk = TimeMix(32, H, D, 4, 1e-6, dt, kind[0])
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    w["w0"] = torch.linspace(-9.0, -3.0, H * D)
    w["norm"] = torch.ones(H * D)
    blk.load({n: t.to(torch.bfloat16) for n, t in w.items()})
    decay = torch.exp(-torch.exp(w["w0"].to(torch.bfloat16).double())).view(H, D)
    for hot in (0, 15, 16, 63, 64, 127):
        val = {n: torch.zeros(T, len(r)) for n, r in blk._rows().items()}
        val["k"][hot], val["v"][hot], val["r"][:], val["g"][:] = 1.0, 2.0, 0.5, 1.0
        proj = packed(blk, T, val, kind)
        for cuts in ([T], [hot + 1, T - hot - 1], [T - 3, 1, 1, 1], [hot + 2, T - hot - 2]):
            got, run, seq = run_core(blk, proj, cuts, kind)
            st = run[1][seq.slot].cpu().double()
            want = 2.0 * decay ** (T - 1 - hot)                 # (the token's own step does not decay it)
            assert ((st[:, 5, :D] - want).abs() < 5e-5 * want + 1e-9).all(), (hot, cuts)
            assert float(got[:hot + 1].abs().sum()) == 0.0      # no bonus: the token itself is not in its read-out
            live = got[hot + 1:, blk._out_columns()]
            assert (live - live[:1]).abs().max() < 0.02 and float(live.min()) > 0.5


SSD_SIZES = [(6, 10, 7, 3, 3, 4), (2, 16, 16, 1, 4, 1), (4, 32, 64, 2, 4, 2), (2, 64, 128, 1, 4, 4), (1, 136, 48, 1, 1, 2), (3, 40, 200, 3, 8, 1),
             (2, 100, 112, 1, 2, 1)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,E,N,G,K,parts", SSD_SIZES)
def test_ssd_alone(kind, H, E, N, G, K, parts):
    dt = getattr(torch, kind[1])
    g = torch.Generator().manual_seed(N)
    T, eps, inner = 141, 1e-2, H * E
    blk = SSD(32, H, E, N, G, K, parts, eps, dt, kind[0])
    blk.out_scale = 1.4
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    C = inner + 2 * G * N
    w.update({"conv": torch.randn(C, K, generator=g) * 0.6, "conv.b": torch.randn(C, generator=g) * 0.5, "D": torch.randn(H, generator=g),
              "dt_bias": torch.randn(H, generator=g) - 1.0, "A_log": torch.linspace(-4.0, 3.0, H), "norm": 1 + 0.3 * torch.randn(inner, generator=g)})
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    d = {n: t.double() for n, t in w.items()}
    val = {"in": torch.randn(T, inner + C + H, generator=g)}
    proj = packed(blk, T, val, kind)
    z = val["in"].to(dt).double()
    xbc = oracle.silu(oracle.causal_conv(z[:, inner:inner + C], d["conv"]) + d["conv.b"])
    x = xbc[:, :inner].view(T, H, E)
    B, Cm = (xbc[:, inner + s * G * N:inner + (s + 1) * G * N].view(T, G, N).repeat_interleave(H // G, dim=1) for s in (0, 1))
    y, S = oracle.ssd_recurrence(x, B, Cm, oracle.softplus(z[:, inner + C:] + d["dt_bias"]), d["A_log"], d["D"])
    want = 1.4 * oracle.gated_group_norm(y.reshape(T, inner), z[:, :inner], d["norm"], parts, eps)
    cols = blk._out_columns()
    tol = 3e-4 if dt == torch.float32 else 0.03
    every = [[T], [64, 1, 63, 13], [1, 2, 15, 1, 16, 17, 89], [2] * 70 + [1], [128] + [1] * 13, [1] * T]
    for cuts in every[:3] if kind[0] == "cpu" else every:
        got, run, seq = run_core(blk, proj, cuts, kind)
        err = (got[:, cols] - want).abs().max(1).values
        assert float(err.max()) < tol * float(want.abs().max()), (cuts[:4], int(err.argmax()))
        rest = [i for i in range(got.shape[1]) if i not in set(cols.tolist())]
        assert float(got[:, rest].abs().sum()) == 0.0
        state = run[1][seq.slot].cpu().double()[:, :E, :N].transpose(1, 2)
        assert (state - S).abs().max() < (1e-4 if dt == torch.float32 else 0.01) * float(S.abs().max()), cuts[:4]


@pytest.mark.parametrize("kind", KINDS)
def test_ssd_keeps_a_far_token(kind):
    """One loud token far back, silence after it: the state holds it at the size its head's decays leave."""
    dt = getattr(torch, kind[1])
    T, H, E, N = 150, 2, 16, 32
    blk = SSD(32, H, E, N, 1, 1, 1, 1e-6, dt, kind[0])
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    w["conv"] += 1.0
    w["norm"] += 1.0
    w["A_log"] = torch.tensor([-4.0, -6.0])
    w["dt_bias"] += 1.0
    blk.load({n: t.to(torch.bfloat16) for n, t in w.items()})
    dt0 = math.log1p(math.exp(1.0))
    amp = float(torch.tensor(2.0 / (1 + math.exp(-2.0))).to(dt))            # silu(2)
    for hot in (0, 15, 16, 63, 64, 127):
        val = torch.zeros(T, 2 * H * E + 2 * N + H)
        val[hot, H * E:2 * H * E + N] = 2.0
        proj = packed(blk, T, {"in": val}, kind)
        for cuts in ([T], [hot + 1, T - hot - 1], [T - 3, 1, 1, 1], [hot + 2, T - hot - 2]):
            _, run, seq = run_core(blk, proj, cuts, kind)
            st = run[1][seq.slot].cpu().double()
            for h, a in enumerate((-4.0, -6.0)):
                want = dt0 * amp * amp * math.exp(-math.exp(a) * dt0 * (T - 1 - hot))
                assert abs(float(st[h, 3, 5]) - want) < 1e-4 * want, (hot, h, cuts)


@pytest.mark.parametrize("kind", KINDS[1:])
@pytest.mark.parametrize("mixer", ["mix", "mix128", "ssd", "ssd_wide"])
def test_long_portions_are_walked_in_spans(kind, mixer):
    """Portions longer than a span (and one just as long, one a token longer), from nothing and from what earlier ones left, beside
    a short one of another sequence."""
    dt, g = getattr(torch, kind[1]), torch.Generator().manual_seed(2)
    T, short = 1085, 70
    if mixer.startswith("mix"):
        H, D = 2, 128 if mixer == "mix128" else 32
        blk = TimeMix(32, H, D, 8, 1e-2, dt, kind[0])
        proj, z, decay, d = mix_case(blk, T, kind, 5, 2.5)
        o, S = oracle.bonus_recurrence(*(z[n].view(T, H, D) for n in "rkv"), decay, d["u"])
        want = oracle.over_rms(o, 1e-2).reshape(T, H * D) * d["norm"] * oracle.silu(z["g"])
    else:
        H, E, N = (2, 24, 32) if mixer == "ssd" else (1, 136, 16)
        blk = SSD(32, H, E, N, 1, 1, 1, 1e-2, dt, kind[0])
        w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
        w.update({"conv": torch.ones(H * E + 2 * N, 1), "norm": torch.ones(H * E), "D": torch.randn(H, generator=g),
                  "dt_bias": torch.full((H,), -1.0), "A_log": torch.linspace(-5.0, -2.0, H)})
        w = {n: t.to(torch.bfloat16) for n, t in w.items()}
        blk.load(w)
        d = {n: t.double() for n, t in w.items()}
        val = torch.randn(T, 2 * H * E + 2 * N + H, generator=g)
        proj, z = packed(blk, T, {"in": val}, kind), val.to(dt).double()
        xbc = oracle.silu(z[:, H * E:-H])
        B, C = (xbc[:, H * E + i * N:H * E + (i + 1) * N][:, None].expand(T, H, N) for i in (0, 1))
        y, S = oracle.ssd_recurrence(xbc[:, :H * E].view(T, H, E), B, C, oracle.softplus(z[:, -H:] + d["dt_bias"]), d["A_log"], d["D"])
        want = oracle.gated_group_norm(y.reshape(T, H * E), z[:, :H * E], d["norm"], 1, 1e-2)
    cols, tol = blk._out_columns(), (3e-4 if dt == torch.float32 else 0.03) * float(want.abs().max())
    for cuts in ([T], [512, 573], [513, 1, 571], [3, 1082]) if kind[0] == "cuda" else ([T],):
        got, run, seq = run_core(blk, proj, cuts, kind)
        err = (got[:, cols] - want).abs().max(1).values
        assert float(err.max()) < tol, (cuts, int(err.argmax()))
        state = run[1][seq.slot].cpu().double().transpose(1, 2)[:, :S.shape[1], :S.shape[2]]
        assert (state - S).abs().max() < (1e-4 if dt == torch.float32 else 0.01) * float(S.abs().max()), cuts
    cache = HybridCache([blk.run_spec()], 200, 8, 2, 1200, dt, kind[0])
    b = RaggedBatch(cache, [(HybridSequence(cache), [0] * short), (HybridSequence(cache), [0] * T)], None, list(blk.masks), 0, list(blk.tiles))
    rows = torch.cat([proj[:short], proj])
    got = blk.core(rows, cache.runs[0], b).float().cpu().double()[:, cols]
    assert (got[:short] - want[:short]).abs().max() < tol and (got[short:] - want).abs().max() < tol


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,vdim,vp,parts", [(4, 8, 8, 1), (4, 8, 8, 4), (6, 5, 8, 5), (2, 512, 512, 2), (64, 64, 64, 1), (3, 100, 104, 12)])
def test_part_norm(kind, heads, vdim, vp, parts):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(vdim)
    T = 5
    y = torch.randn(T, heads, vdim, generator=g).to(dt)
    wt = 1 + 0.3 * torch.randn(heads, vdim, generator=g)
    t, weight = torch.zeros(T, heads * vp + 8, dtype=dt), torch.zeros(heads, vp)
    t[:, :heads * vp].view(T, heads, vp)[..., :vdim] = y
    weight[:, :vdim] = wt
    z = torch.randn(T, heads * vp + 16, generator=g).to(dt)
    for gate in (None, z):
        wide = t.clone().to(dev)
        part_norm_(wide, gate.to(dev) if gate is not None else None, weight.reshape(-1).to(dev), heads, vdim, vp, parts, 1e-2, 0.6)
        v = y.double()
        if gate is not None:
            v = v * oracle.silu(z[:, :heads * vp].double().view(T, heads, vp)[..., :vdim])
        want = 0.6 * oracle.over_rms(v.reshape(T, parts, -1), 1e-2).view(T, heads, vdim) * wt.double()
        got = wide.cpu().double()
        assert (got[:, :heads * vp].view(T, heads, vp)[..., :vdim] - want).abs().max() < (1e-5 if dt == torch.float32 else 0.03)
        assert float(got[:, heads * vp:].abs().sum()) == 0.0


# ---------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer(kind, name):
    toks = tokens_for(CONFIGS[name], 41)
    trace = []
    want = oracle.run_model(CONFIGS[name], weights_of(name), toks, trace=trace)
    eng = engine_for(name, kind)
    seen = []
    b = eng.model.make_batch(eng.cache, [(eng.open(), toks)], [range(41)])
    got = eng.model.forward_ragged(b, eng.cache, on_layer=lambda r, x: seen.append((r, x.cpu().double())))
    check(got, want, kind, "logits")
    assert [r for r, _ in seen] == list(range(len(trace)))
    for (r, x), t in zip(seen, trace):
        assert float(row_error(x, t).max()) < TOL[getattr(torch, kind[1])], f"residual after layer {r}"
    assert got.dtype == torch.float32


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_decoding_agree_with_the_whole(kind, name):
    toks = tokens_for(CONFIGS[name], 46)
    want = reference(name, toks)
    eng = engine_for(name, kind, blocks=8)
    for cuts in ([1] * 46, [2] * 23, [3, 2, 1, 7, 16, 1, 2, 13, 1], [31] + [1] * 15, [1, 45]):
        seq = eng.open()
        check(feed(eng, seq, toks, cuts), want, kind, str(cuts[:5]))
        eng.close(seq)                            # the next form runs on the pages and the slot of this one
    assert eng.allocated_blocks() == 0 and eng.cache.slot_allocator.num_used() == 0


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("graph", [True, False])
@pytest.mark.parametrize("name", ["odd", "plain"])
def test_mixed_batches_equal_each_alone(kind, graph, name):
    """Portions beside single tokens, requests that pause, end and give their pages and slot to others."""
    lens = {"a": 40, "b": 23, "c": 9, "d": 31, "e": 17}
    toks = {i: tokens_for(CONFIGS[name], n, seed=ord(i)) for i, n in lens.items()}
    want = {i: reference(name, t) for i, t in toks.items()}
    eng = engine_for(name, kind, blocks=18, block=8, batch=4, use_cuda_graph=graph)
    plan = [{"a": 11, "b": 2}, {"a": 1, "b": 1, "c": 3}, {"a": 1, "b": 1, "c": 1}, {"c": 5, "b": 19, "d": 1}, {"d": 2}, {"d": 1, "a": 13},
            {"d": 1, "a": 1, "e": 2}, {"a": 13, "e": 1, "d": 1}, {"e": 14, "d": 25}]
    live, at = {}, dict.fromkeys(lens, 0)
    for step in plan:
        entries = []
        for i, n in step.items():
            live.setdefault(i, eng.open())
            entries.append((live[i], toks[i][at[i]:at[i] + n]))
        got = eng.execute(entries, [list(range(n)) for n in step.values()]).cpu()
        row = 0
        for i, n in step.items():
            check(got[row:row + n], want[i][at[i]:at[i] + n], kind, f"{i} from {at[i]}")
            row += n
            at[i] += n
            if at[i] == lens[i]:
                eng.close(live.pop(i))
    assert at == lens and eng.allocated_blocks() == 0


@pytest.mark.parametrize("kind", KINDS)
def test_long_prompt_and_long_decoding(kind):
    """Across chunks, key tiles, windows and splits: a prompt of 300 tokens in unequal portions, then decoding."""
    name = "plain"
    toks = tokens_for(CONFIGS[name], 420)
    want = reference(name, toks)
    eng = engine_for(name, kind, blocks=54)
    check(feed(eng, eng.open(), toks, [270, 30] + [1] * 120), want, kind)
    eng = engine_for(name, kind, blocks=54)
    check(feed(eng, eng.open(), toks, [5, 65, 256, 94]), want, kind)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["attention", "mixing", "dual"])
def test_far_and_first_tokens_reach_the_logits(kind, name):
    toks = tokens_for(CONFIGS[name], 30)
    other = [(toks[0] + 1) % CONFIGS[name]["vocab"]] + toks[1:]
    a, b = reference(name, toks), reference(name, other)
    assert float(row_error(a[-1:], b[-1:]).max()) > 20 * TOL[torch.float32]
    for t, w in ((toks, a), (other, b)):
        eng = engine_for(name, kind)
        check(feed(eng, eng.open(), t, [1, 2, 26, 1]), w, kind)


def test_wanted_rows_come_in_entry_order_and_nothing_is_kept_of_a_refused_step():
    eng = engine_for("odd", ("cpu", "float32"), blocks=5, block=8, batch=2)
    ta, tb = tokens_for(CONFIGS["odd"], 12, 3), tokens_for(CONFIGS["odd"], 20, 4)
    a, b = eng.open(), eng.open()
    got = eng.execute([(a, ta), (b, tb[:1])], [[11, 2], [0]])
    check(got, torch.stack([reference("odd", ta)[11], reference("odd", ta)[2], reference("odd", tb)[0]]), ("cpu", "float32"))
    assert eng.execute([(b, tb[1:3])], [[]]) is None
    with pytest.raises(RuntimeError, match="KV blocks"):
        eng.execute([(a, [1]), (b, tb[3:] + [0] * 20)], [[0], [0]])
    check(eng.execute([(b, tb[3:])], [range(17)]), reference("odd", tb)[3:], ("cpu", "float32"))


# ---------------------------------------------------------------------------------------- generation
def greedy(name, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(oracle.run_model(CONFIGS[name], weights_of(name), out)[-1].argmax()))
    return out


@pytest.mark.parametrize("kind", [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu)])
def test_greedy_generation_through_every_entry_point(kind):
    name = "odd"
    prompts = [tokens_for(CONFIGS[name], n, seed=n) for n in (3, 12, 1, 9, 12)]
    want = [greedy(name, p, 9) for p in prompts]
    gen = GenerateConfig(max_new_tokens=9)
    m = make_model(CONFIGS[name], weights_of(name), kind)
    assert m.generate(prompts[1], gen) == want[1]
    # the engine: a step budget that cuts prompts, fewer slots than requests, pages that run short
    for budget, blocks in ((5, 64), (8192, 6)):
        eng = make_engine(m, EngineConfig(block_size=8, num_blocks=blocks, max_seq_len=48, max_batch_size=3), max_step_tokens=budget)
        assert isinstance(eng, HybridEngine)
        ids = [eng.add_request(p, gen) for p in prompts]
        eng.run()
        assert [eng.result(i) for i in ids] == want
        assert eng.allocated_blocks() == 0 and eng._promised == 0
    sch = ContinuousBatchingScheduler(m, EngineConfig(block_size=8, num_blocks=32, max_seq_len=48, max_batch_size=3))
    ids = [sch.add_request(p, gen) for p in prompts]
    sch.run()
    assert [sch.result(i) for i in ids] == want


def test_sampling_and_presets():
    cfg = vobotar.preset("tiny", torch.float32)
    m = HybridModel(cfg, init_std=0.1, seed=3)
    p = tokens_for({"vocab": cfg.vocab_size}, 6)
    gen = GenerateConfig(max_new_tokens=8, do_sample=True, seed=11)
    out = m.generate(p, gen)
    assert len(out) == 14 and out == m.generate(p, gen)
    assert vobotar.preset("small", torch.bfloat16).vocab_size == 4096
    with pytest.raises(ValueError, match="preset"):
        vobotar.preset("huge", torch.float32)


# ---------------------------------------------------------------------------------------- files, registry, replay
def write_model(folder, name, config=None):
    from tesseract_b200.io.safetensors import save_file
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config or CONFIGS[name]))
    save_file(weights_of(name), str(folder / "model.safetensors"), {})


@pytest.mark.parametrize("name", ["odd", "wide"])
def test_registry_files_and_round_trip(tmp_path, name):
    write_model(tmp_path / "m", name)
    m = load_pretrained(str(tmp_path / "m"), torch.float32, "cpu")
    assert isinstance(m, HybridModel) and m.config.architecture == "Vobotar"
    arch = resolve(CONFIGS[name])
    from tesseract_b200.build import GROUPS
    assert arch.name == "Vobotar" and arch.kernels in GROUPS
    assert vobotar.config_to_dict(m.config) == CONFIGS[name]
    for k, t in m.state_tensors().items():
        assert torch.equal(t.to(torch.bfloat16), weights_of(name)[k]), k
    m.save_safetensors(str(tmp_path / "copy.safetensors"))
    again = HybridModel(m.config)
    assert again.load_safetensors(str(tmp_path / "copy.safetensors")) == []
    assert sum(t.numel() for t in m.parameters()) >= sum(t.numel() for t in weights_of(name).values())
    sd = dict(weights_of(name))
    for k in ("embed", "side.embed", "l0.norm1", "final.norm", "l0.side.proj", *(("l0.mix.vmix", "l1.mix.left.sink", "l1.mix.right.mu.w",
              "l2.mix.right.conv.b", "l2.mix.left.k.norm", "l0.mlp.up") if name == "odd" else ())):
        with pytest.raises(KeyError, match="missing"):
            m.load_tensors({n: t for n, t in sd.items() if n != k})
    key = next(k for k in sd if k.startswith("l1.mix") and k.endswith("o"))
    sd[key] = sd[key][:, 1:]
    with pytest.raises(ValueError, match="l1.mix"):
        m.load_tensors(sd)


def test_the_decays_inputs_may_only_be_in_the_weights(tmp_path):
    config = json.loads(json.dumps(CONFIGS["mixing"]))
    for l in config["layers"]:
        l["mixer"]["right"].pop("rank")
    write_model(tmp_path / "m", "mixing", config)
    m = load_pretrained(str(tmp_path / "m"), torch.float32, "cpu")
    assert [l.mixer.right.rank for l in m.config.layers] == [4, 9]
    toks = tokens_for(config, 20)
    check(m.forward(torch.tensor([toks]))[0], reference("mixing", toks), ("cpu", "float32"))


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="ring"), "mixer"), (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["layers"][0]["mixer"].pop("softcap"), "softcap"), (lambda c: c.pop("token_side"), "token_side"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "rotary"), (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "mask.size")])
def test_config_errors(change, what):
    c = json.loads(json.dumps(CONFIGS["odd"]))
    change(c)
    with pytest.raises(ValueError, match=what):
        vobotar.config_from_dict(c)


def test_size_errors():
    bf = torch.bfloat16
    for bad in (lambda: AttentionGeometry(3, 2, 8, 8, bf), lambda: AttentionGeometry(1, 1, 264, 8, bf), lambda: AttentionGeometry(1, 1, 8, 6, bf, None, True),
                lambda: AttentionGeometry(1, 1, 8, 8, bf, gate="both"), lambda: Window(0), lambda: TimeMixGeometry(2, 260, 8), lambda: TimeMixGeometry(2, 8, 0),
                lambda: SSDGeometry(3, 8, 8, 2, 4, 1), lambda: SSDGeometry(2, 8, 264, 1, 4, 1), lambda: SSDGeometry(2, 8, 8, 1, 9, 1),
                lambda: SSDGeometry(2, 9, 8, 1, 4, 4)):
        with pytest.raises(ValueError):
            bad()
    a = ShapedAttentionSpec(1, 1, 8, 8, 1.0, v_mix=True)
    mix = SideBySideSpec(TimeMixSpec(1, 8, 4), ShapedAttentionSpec(1, 1, 8, 8, 1.0))
    for kw in (dict(layers=[LayerSpec(a, SiluGLUSpec(8))], form="parallel"), dict(layers=[LayerSpec(a)], token_side=4),
               dict(layers=[LayerSpec(a), LayerSpec(ShapedAttentionSpec(1, 1, 8, 4, 1.0, v_mix=True))], form="post"),
               dict(layers=[LayerSpec(mix)], form="post"), dict(layers=[LayerSpec(a, GLUSpec(8, 1.0))], form="post")):
        with pytest.raises(ValueError):
            HybridModel(HybridConfig(8, 8, **kw))


@pytest.mark.parametrize("kind", KINDS)
def test_mixers_also_run_alone_and_in_sandwich_layers(kind):
    """The same mixers, side by side and each alone, between Dynamic Tanh norms: prompts against decoding."""
    src = vobotar.config_from_dict(CONFIGS["plain"], getattr(torch, kind[1]))
    mixers = [s.mixer for s in src.layers] + [TimeMixSpec(2, 16, 8), SSDSpec(4, 16, 16, 2, 3, 2)]
    layers = [LayerSpec(m, SiluGLUSpec(24) if i % 2 else GLUSpec(24, 2.0)) for i, m in enumerate(mixers) if not getattr(m, "v_mix", False)]
    m = HybridModel(HybridConfig(40, 48, layers, dtype=src.dtype), device=kind[0], init_std=0.2, seed=4)
    toks = tokens_for({"vocab": 40}, 70, 5)
    whole = m.forward(torch.tensor([toks]))[0].float().cpu()
    eng = HybridEngine(m, EngineConfig(block_size=8, num_blocks=16, max_seq_len=128, max_batch_size=2))
    check(feed(eng, eng.open(), toks, [40, 3, 7] + [1] * 20), whole, kind)


@pytest.mark.parametrize("kind", KINDS)
def test_trace_replay(kind, tmp_path):
    from tesseract_b200.serving.trace import make_replay, replay
    write_model(tmp_path / "m", "odd")
    ta, tb = tokens_for(CONFIGS["odd"], 25, 8), tokens_for(CONFIGS["odd"], 30, 9)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ta[:20], "want": [0, 19]}, {"id": "y", "tokens": tb[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": tb[3:5], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": tb[5:6], "want": [0]}, {"id": "x", "tokens": ta[20:], "want": [4]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": tb[6:], "want": [23]}, {"id": "x", "tokens": tb[:1], "want": [0]}], "end": ["x", "y"]}]
    rep = make_replay(str(tmp_path / "m"), getattr(torch, kind[1]), torch.device(kind[0]), 64)
    said = []
    replay(rep, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(4)]
    ra, rb = reference("odd", ta), reference("odd", tb)
    for n, rows in {0: [ra[0], ra[19]], 2: [rb[5], ra[24]], 3: [rb[29], rb[0]]}.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(len(rows), -1))
        check(got, torch.stack(rows), kind, f"step {n}")
    assert rep.engine.allocated_blocks() == 0 and rep.live == {}


@pytest.mark.gpu
def test_padding_rows_of_a_captured_step_touch_nothing():
    """Three sequences decode in a bucket of four: the padding row leaves every page and slot alone."""
    eng = engine_for("plain", ("cuda", "bfloat16"), blocks=24, batch=4)
    toks = [tokens_for(CONFIGS["plain"], 12, s) for s in range(3)]
    seqs = [eng.open() for _ in toks]
    eng.execute([(s, t[:11]) for s, t in zip(seqs, toks)], [[], [], []])
    eng.warm_graphs()
    used = {b for s in seqs for b in s.blocks}
    keep = {24: [b for b in range(24) if b not in used], 4: [3]}
    stores = [t for r in eng.cache.runs for t in eng.cache.tensors(r)]
    before = [t.clone() for t in stores]
    got = eng.execute([(s, t[11:]) for s, t in zip(seqs, toks)], [[0]] * 3)
    assert 4 in eng._graphs
    for now, was in zip(stores, before):
        rows = keep.get(now.shape[0], slice(None))              # (the angles do not change either)
        assert torch.equal(now[rows], was[rows])
    check(got, torch.stack([reference("plain", t)[11] for t in toks]), ("cuda", "bfloat16"))


@pytest.mark.gpu
def test_kernels_report_no_status():
    from tesseract_b200 import _native
    n0 = _native.launch_count()
    eng = engine_for("wide", ("cuda", "bfloat16"))
    feed(eng, eng.open(), tokens_for(CONFIGS["wide"], 20), [17, 1, 2])
    assert _native.launch_count() > n0
    assert _native.read_status(torch.cuda.current_stream().cuda_stream) == 0

"""Polosun (latent attention, retention, real-gated recurrence, side-by-side sublayers, depth averaging) against the plain
statements of ``polosun_oracle``: every mechanism alone, prompts, portions, batches, decoding, reuse of pages and slots,
and generation through the framework's entry points. The same tests run on the CPU and, marked ``gpu``, on the kernels."""
import io
import json
import math

import numpy as np
import pytest
import torch

import polosun_oracle as oracle
from tesseract_b200 import ops
from tesseract_b200.models import GenerateConfig, load_pretrained, polosun
from tesseract_b200.models.hybrid import (AttentionSpec, GLUSpec, HybridConfig, HybridModel, LayerSpec, SiluGLUSpec)
from tesseract_b200.models.registry import resolve
from tesseract_b200.models.scheduler import ContinuousBatchingScheduler, EngineConfig
from tesseract_b200.nn.hybrid import RGLRU, LatentAttention, Retention
from tesseract_b200.nn.ragged import HybridCache, HybridSequence, RaggedBatch
from tesseract_b200.ops.latent import LatentGeometry
from tesseract_b200.ops.retention import RetentionGeometry, log2_decays
from tesseract_b200.ops.rglru import RGLRUGeometry
from tesseract_b200.ops.rotary import Rotary, Yarn
from tesseract_b200.serving import HybridEngine, make_engine

KINDS = [("cpu", "float32"), ("cpu", "bfloat16"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu),
         pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]
# relative error of a row of logits: bf16 rounding alone reaches 0.03 in single rows; a mechanism that is off by one token
# or factor shows as 0.3 and more
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.1}
MEAN_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.03}


def latent(heads, dim, rot, vdim, rank, scale, base=1e4, scaling=None, ff=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                                                  "scale": scale, "rot": r}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def ret(heads, dim, vdim, decay, dims, base=1e4, ff=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"base": base, "dims": dims}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def rec(width, blocks, conv, ff=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def conf(vocab, width, layers, mult=0.7, eps=1e-5):
    return {"architecture": "Polosun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult}


CONFIGS = {
    # sizes that are multiples of nothing, layers without a feed-forward, partly rotated heads, extreme decays
    "odd": conf(53, 42, [ret(3, 11, 7, (0.8, 0.93, 1.0), 6, 100.0, 27), latent(5, 7, 6, 9, 13, 0.4, 50.0, (3.0, 16, 4.0, 0.5), 30), rec(21, 3, 4),
                         latent(2, 10, 4, 5, 20, 0.7), rec(40, 1, 1, 18), ret(2, 9, 10, (0.8, 0.95), 0)], 1.0, 1e-3),
    # even sizes, two of each
    "plain": conf(130, 96, [rec(96, 4, 3, 72), ret(2, 64, 64, (0.9, 0.98), 64, 1e4, 80), latent(3, 32, 32, 64, 64, 0.2, 1e4, None, 64), ret(4, 32, 16,
                            (0.8, 0.95, 0.99, 0.999), 16, 1e3), latent(4, 64, 16, 48, 96, 0.15, 1e4, (8.0, 32, 8.0, 1.0), 48), rec(64, 2, 2, 40)], 0.6, 1e-6),
    # more than sixteen heads; heads and a latent too large for the fast kernels; values wider than a tile
    "wide": conf(64, 128, [latent(20, 64, 64, 128, 128, 0.09, 1e6, None, 96), ret(1, 200, 24, (0.97,), 100), ret(2, 48, 264, (0.9, 0.99), 48, 1e4, 64),
                           latent(2, 100, 60, 40, 544, 0.08)], 0.9),
    # attention only, recurrence only
    "latent": conf(33, 32, [latent(2, 16, 8, 16, 24, 0.3, 1e4, None, 24), latent(4, 8, 16, 12, 64, 0.3)], 1.3, 1e-4),
    "state": conf(40, 48, [ret(2, 16, 24, (0.995, 0.97), 8, 1e4, 24), rec(48, 3, 5)], 0.8, 1e-4),
}


def make_weights(config, seed=0):
    """bf16 tensors for every name the model has, sized so that no mechanism fades."""
    g = torch.Generator().manual_seed(seed)
    model = HybridModel(polosun.config_from_dict(config))

    def draw(name, shape):
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if shape == ():
            return 0.7 + 0.6 * torch.rand((), generator=g)          # the gains differ from one another and from 1
        if last == "dwa":
            return torch.cat([0.4 * r[:-1], 1.0 + 0.2 * r[-1:]])
        if last == "lam":
            return 1.5 * r - 2.5
        if last == "conv":
            return r * 0.6
        if last == "b":
            return 0.4 * r
        if len(shape) == 1:
            return 1.0 + 0.3 * r
        return r * (1.5 / math.sqrt(shape[-1]))
    w = {n: draw(n, s) for n, s in model.logical_shapes().items()}
    for i, l in enumerate(config["layers"]):
        if l["type"] == "retention":          # the read-out over its own size has the sign of q . k: keep that away from zero
            w[f"l{i}.mix.k"] = 0.8 * w[f"l{i}.mix.q"] + 0.6 * w[f"l{i}.mix.k"]
    return {n: t.to(torch.bfloat16) for n, t in w.items()}


def make_model(config, weights, kind):
    m = HybridModel(polosun.config_from_dict(config, getattr(torch, kind[1])), device=kind[0])
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
    if len(e) >= 8:
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
@pytest.mark.parametrize("dims,base,scaling", [(64, 1e4, None), (12, 5e5, (4.0, 1024, 32.0, 1.0)), (6, 50.0, (3.0, 16, 4.0, 0.5)),
                                               (2, 9.0, (2.0, 64, 1000.0, 0.001)), (16, 1e4, (8.0, 4096, 0.25, 0.25))])
def test_rotary_frequencies_layout_and_far_positions(dims, base, scaling):
    r = Rotary(dims, base, Yarn(*scaling) if scaling else None)
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    f, mult = oracle.rotary_frequencies(rot)
    table = r.table(70000)                                     # (longer than one piece of the computation)
    for p in (0, 1, 777, 65535, 65536, 69999):
        for i in range(dims // 2):
            assert abs(float(table[p, i, 0]) - mult * math.cos(p * f[i])) < 2e-7 * mult
            assert abs(float(table[p, i, 1]) - mult * math.sin(p * f[i])) < 2e-7 * mult
    dim = dims + 5
    cols = r.columns(dim).tolist()
    assert len(set(cols)) == dim and max(cols) < r.stored(dim) and r.stored(dim) % 8 == 0
    for i in range(dims // 2):
        assert cols[i + dims // 2] - cols[i] == r.hp
    x = torch.randn(3, 2, dim, dtype=torch.float64)
    stored = torch.zeros(3, 2, r.stored(dim))
    stored[..., cols] = x.float()
    from tesseract_b200.ops.rotary import rotate_stored
    got = rotate_stored(stored, table, torch.tensor([5, 0, 900]))[..., cols]
    assert (got - oracle.rotate(x, [5, 0, 900], rot)).abs().max() < 1e-5


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("W,cols", [(40, 48), (37, 48), (256, 256), (1030, 1040), (2304, 2304)])
def test_depth_residual_in_every_form(kind, W, cols):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(W)
    T, V, eps = 11, 19, 1e-3
    rnd = lambda *s: torch.randn(*s, generator=g)   # noqa: E731
    table = torch.zeros(V, cols, dtype=dt)
    table[:, :W] = rnd(V, W)
    toks = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    emb = table[toks.long(), :W].double()
    htol = 3e-5 if dt == torch.float32 else 0.03

    def is_norm(h, x, gain):
        want = oracle.scalar_rms_norm(x.double(), gain, eps)
        assert (h[:, :W].cpu().double() - want).abs().max() < htol and float(h[:, W:].abs().sum()) == 0.0
    # start of the model, with and without a history
    hist = torch.zeros(3, T, W, device=dev)
    x, h = ops.depth_residual(tokens=toks.to(dev), table=table.to(dev), width=W, history=hist, gain=0.6, eps=eps, out_cols=cols, out_dtype=dt)
    assert torch.equal(x.cpu().double(), emb) and torch.equal(hist[0].cpu().double(), emb)
    is_norm(h, emb, 0.6)
    x, h = ops.depth_residual(tokens=toks.to(dev), table=table.to(dev), width=W, eps=eps, out_cols=cols, out_dtype=dt)
    assert torch.equal(x.cpu().double(), emb)
    is_norm(h, emb, 1.0)
    # a step: plain, averaged over one and over two earlier entries, stored or not
    x0, y = rnd(T, W), (2 * rnd(T, W)).to(dt)
    new = x0.double() + 0.35 * y.double()
    x, h = ops.depth_residual(x0.to(dev), y.to(dev), 0.35, gain=1.4, eps=eps, out_cols=cols, out_dtype=dt)
    assert (x.cpu().double() - new).abs().max() < 1e-5
    is_norm(h, new, 1.4)
    past = rnd(2, T, W)
    for depth, store in ((1, True), (2, True), (2, False)):
        hist = torch.zeros(3, T, W, device=dev)
        hist[:2] = past.to(dev)
        avg = rnd(depth + 1)
        want = oracle.depth_average([*past[:depth].double(), new], avg.double())
        x, h = ops.depth_residual(x0.to(dev), y.to(dev), 0.35, history=hist, depth=depth, average=avg.to(dev), store=store, eps=eps,
                                  out_cols=cols, out_dtype=dt)
        assert (x.cpu().double() - want).abs().max() < 2e-5                # the residual stays in 32-bit whatever the type
        is_norm(h, want, 1.0)
        stored = new if store else (past[depth].double() if depth < 2 else torch.zeros(T, W))
        assert (hist[depth].cpu().double() - stored).abs().max() < 1e-5


@pytest.mark.parametrize("kind", KINDS)
def test_silu_glu_scales_both_halves_and_writes_into_columns(kind):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(0)
    F = 48
    gu = (3 * torch.randn(9, 2 * F, generator=g)).to(dt)
    gu[0, :8] = torch.tensor([-200.0, 200.0, -20.0, 20.0, 0.0, -1.0, 1.0, -90.0])
    z = 0.7 * gu.double()
    want = oracle.silu(z[:, :F]) * z[:, F:]
    wide = torch.full((9, F + 16), 5.0, dtype=dt, device=dev)
    ops.silu_glu(gu.to(dev), 0.7, wide[:, 16:])
    got = wide.cpu().double()
    assert ((got[:, 16:] - want).abs() < (1e-5 if dt == torch.float32 else 0.01) * want.abs().clamp_min(1.0)).all()
    assert bool((got[:, :16] == 5.0).all())


def packed(block, T, values, kind):
    """The block's packed projection rows with the given logical values."""
    p = torch.zeros(T, block.cols)
    for name, rows in block._rows().items():
        p[:, rows] = values[name].reshape(T, -1).float()
    return p.to(getattr(torch, kind[1])).to(kind[0])


def run_core(block, proj, cuts, kind, block_size=8, dirty=True, before=0):
    """Feeds rows of ``proj`` through a cache of one sequence whose slot and pages hold what an earlier one left."""
    T = proj.shape[0]
    n = (T + block_size - 1) // block_size
    cache = HybridCache([block.run_spec()], n + 3, block_size, 2, (n + 3) * block_size, block.dtype, kind[0])
    run = cache.runs[0]
    rotary = 0 if isinstance(block, RGLRU) else 1
    if dirty:
        for t in run[:len(run) - rotary]:
            t.copy_(torch.randn(t.shape).to(t.dtype))
    cache.allocator.allocate()                   # the sequence's pages and slot are not the pool's first
    cache.slot_allocator.allocate()
    seq, got, at = HybridSequence(cache), [], 0
    for n in cuts:
        b = RaggedBatch(cache, [(seq, [0] * n)], None, [0], 0, [block.tile] if block.tile else [])
        got.append(block.core(proj[at:at + n].contiguous(), run, b).float().cpu())
        b.commit()
        at += n
    assert at == T
    return torch.cat(got).double(), run, seq


LATENT_SIZES = [(3, 12, 8, 10, 20), (16, 64, 64, 128, 512), (18, 32, 32, 64, 64), (2, 100, 60, 36, 48), (2, 24, 16, 150, 576)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,D,R,E,C", LATENT_SIZES)
def test_latent_attention_alone(kind, H, D, R, E, C):
    dt = getattr(torch, kind[1])
    g = torch.Generator().manual_seed(H * C)
    T, eps, scale = 37, 1e-2, 1.5 * (D + R) ** -0.5
    rot = {"dims": R, "base": 100.0, "scaling": {"factor": 2.5, "original": 24, "fast": 3.0, "slow": 0.5}}
    blk = LatentAttention(32, H, D, R, E, C, scale, Rotary(R, 100.0, Yarn(2.5, 24, 3.0, 0.5)), eps, dt, kind[0])
    w = {"dkv.norm": 1 + 0.3 * torch.randn(C, generator=g), "uk": torch.randn(H * D, C, generator=g) * C ** -0.5,
         "uv": torch.randn(H * E, C, generator=g) * C ** -0.5}
    for n, s in blk.logical_shapes().items():
        w.setdefault(n, torch.zeros(s))
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    blk.in_scale = 0.8
    val = {n: torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
    val["dkv"] = val["dkv"] * 0.2                # (the latent's mean square is near eps: where eps goes shows)
    proj = packed(blk, T, val, kind)
    z = {n: 0.8 * v.to(dt).double() for n, v in val.items()}
    q = z["q"].view(T, H, D + R)
    c = oracle.over_rms(z["dkv"][:, :C], eps) * w["dkv.norm"].double()
    want = oracle.latent_attention(q[..., :D], oracle.rotate(q[..., D:], range(T), rot), c, oracle.rotate(z["dkv"][:, C:], range(T), rot),
                                   w["uk"].double().view(H, D, C), w["uv"].double().view(H, E, C), scale)
    want = (want.reshape(T, H * E) * oracle.sigmoid(z["g"]))
    cols = blk._out_columns()
    for cuts in ([T], [1] * T, [2] * 18 + [1], [17, 1, 1, 16, 2], [1, 36]):
        got, _, _ = run_core(blk, proj, cuts, kind)
        assert (got[:, cols] - want).abs().max() < (1e-4 if dt == torch.float32 else 0.03), cuts[:4]
        rest = [i for i in range(got.shape[1]) if i not in set(cols.tolist())]
        assert float(got[:, rest].abs().sum()) == 0.0


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,D,R,E,C", [(3, 12, 8, 10, 20), (17, 64, 32, 64, 128), (2, 100, 60, 36, 48)])
def test_one_standing_out_key_everywhere(kind, H, D, R, E, C):
    """One key is made to win wherever it is seen, and its value to be unmistakable: every query from it on returns that value,
    no query before it does -- with the key first, last, and on either side of page and key-tile edges."""
    dt = getattr(torch, kind[1])
    g = torch.Generator().manual_seed(C)
    T = 150
    blk = LatentAttention(32, H, D, R, E, C, 1.0, Rotary(R, 1e4), 1e-6, dt, kind[0])
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    w["dkv.norm"] = torch.ones(C)
    w["uk"] = 0.02 * torch.randn(H * D, C, generator=g)
    w["uk"].view(H, D, C)[:, 0, 0] = 1.0                         # coordinate 0 of every key is the latent's coordinate 0
    w["uv"] = 0.1 * torch.randn(H * E, C, generator=g)
    w["uv"].view(H, E, C)[:, :, 0] = 2.0
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    for hot in (0, 7, 8, 63, 64, 127, 128, T - 1):
        val = {n: 0.05 * torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
        val["q"].view(T, H, D + R)[:, :, 0] = 6.0
        val["dkv"][:, 0] = 0.0
        val["dkv"][hot, 0] = 50.0
        val["g"][:] = 20.0
        proj = packed(blk, T, val, kind)
        z = {n: v.to(dt).double() for n, v in val.items()}
        q = z["q"].view(T, H, D + R)
        rot = {"dims": R, "base": 1e4}
        want = oracle.latent_attention(q[..., :D], oracle.rotate(q[..., D:], range(T), rot), oracle.over_rms(z["dkv"][:, :C], 1e-6),
                                       oracle.rotate(z["dkv"][:, C:], range(T), rot), w["uk"].double().view(H, D, C),
                                       w["uv"].double().view(H, E, C), 1.0).reshape(T, H * E)
        top = 2.0 * math.sqrt(C)
        assert (want[hot:] - top).abs().max() < 0.1 * top and (hot == 0 or float(want[:hot].abs().max()) < 0.3 * top)
        for cuts in ([T], [hot + 1] + [1] * min(9, T - hot - 1) + [T - hot - 1 - min(9, T - hot - 1)], [max(hot, 1), 2, T - max(hot, 1) - 2]):
            cuts = [n for n in cuts if n > 0]
            if sum(cuts) != T:
                continue
            got, _, _ = run_core(blk, proj, cuts, kind, block_size=16)
            assert (got[:, blk._out_columns()] - want).abs().max() < (1e-4 if dt == torch.float32 else 0.02) * top, (hot, cuts[:3])


RET_SIZES = [(2, 16, 24, 16), (3, 11, 7, 6), (1, 64, 64, 64), (2, 128, 128, 128), (1, 200, 40, 60), (2, 40, 200, 0)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,D,E,dims", RET_SIZES)
def test_retention_alone(kind, H, D, E, dims):
    """Chunks of 64, spans of 256 and the one-token form against the token-by-token statement, with slow, fast and extreme
    decays; the slot had been used before; the state stays in 32-bit."""
    dt = getattr(torch, kind[1])
    g = torch.Generator().manual_seed(D)
    T, eps = 333, 1e-2
    decay = [(0.999, 0.9, 0.0), (0.97, 1.0, 0.5)][D % 2][:H] if H > 1 else (0.995,)
    blk = Retention(32, H, D, E, decay, Rotary(dims, 300.0), eps, dt, kind[0])
    blk.in_scale = 1.2
    val = {n: torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
    proj = packed(blk, T, val, kind)
    z = {n: 1.2 * v.to(dt).double() for n, v in val.items()}
    rot = {"dims": dims, "base": 300.0}
    q = oracle.rotate(z["q"].view(T, H, D), range(T), rot)
    k = oracle.rotate(z["k"].view(T, H, D), range(T), rot) * D ** -0.5
    o, S = oracle.retention(q, k, z["v"].view(T, H, E), decay)
    want = oracle.over_rms(o, eps).reshape(T, H * E) * oracle.silu(z["g"])
    cols = blk._out_columns()
    tol = 3e-4 if dt == torch.float32 else 0.04
    every = [[T], [64, 1, 191, 77], [1, 2, 254, 76], [255, 1, 1, 76], [300] + [1] * 33]
    for cuts in every[:3] if kind[0] == "cpu" else every + [[1] * T]:
        got, run, seq = run_core(blk, proj, cuts, kind)
        err = (got[:, cols] - want).abs().max(1).values
        assert float(err.max()) < tol * float(want.abs().max()), (cuts[:4], int(err.argmax()))
        state = run[0][seq.slot].cpu().double()[:, blk.geo.rotary.columns(D)][..., :E]
        assert (state - S).abs().max() < (1e-4 if dt == torch.float32 else 0.006) * float(S.abs().max()), cuts[:4]


@pytest.mark.parametrize("kind", KINDS)
def test_retention_keeps_a_far_token(kind):
    """Everything is silent but one token far back: its trace comes out at the size its decay leaves, across chunks, spans and
    portions. (Read before the norm hides sizes: through the state.)"""
    dt = getattr(torch, kind[1])
    T, H, D, E = 290, 2, 16, 8
    decay = (0.99, 0.9975)
    blk = Retention(32, H, D, E, decay, Rotary(0, 10.0), 1e-6, dt, kind[0])
    for hot in (0, 63, 64, 255, 256):
        val = {n: torch.zeros(T, len(r)) for n, r in blk._rows().items()}
        val["k"][hot], val["v"][hot], val["q"][:], val["g"][:] = 1.0, 2.0, 0.5, 1.0
        proj = packed(blk, T, val, kind)
        for cuts in ([T], [hot + 1, T - hot - 1], [T - 3, 1, 1, 1]):
            got, run, seq = run_core(blk, proj, cuts, kind)
            st = run[0][seq.slot].cpu().double()
            for h in range(H):
                want = decay[h] ** (T - 1 - hot) * 2.0 * D ** -0.5
                assert abs(float(st[h, 3, 5]) - want) < 2e-5 * want + 1e-9, (hot, h, cuts)
            live = got[hot:, blk._out_columns()]
            assert (live - live[:1]).abs().max() < 0.02 and float(live.min()) > 0.5
            assert float(got[:hot].abs().sum()) == 0.0


REC_SIZES = [(24, 3, 3), (33, 1, 4), (160, 2, 1), (320, 4, 2), (30, 5, 9)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("W,N,K", REC_SIZES)
def test_rglru_alone(kind, W, N, K):
    dt = getattr(torch, kind[1])
    g = torch.Generator().manual_seed(W)
    T = 139
    blk = RGLRU(32, W, N, K, dt, kind[0])
    shapes = blk.logical_shapes()
    w = {n: torch.randn(s, generator=g) * (0.5 if "conv" in n else W ** -0.5 * N ** 0.5 if len(s) == 3 else 0.5) for n, s in shapes.items()}
    w["lam"] = torch.linspace(-12.0, 9.0, W)                 # decays from nearly none to nearly all
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    blk.in_scale = 0.9
    val = {n: torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
    proj = packed(blk, T, val, kind)
    z = {n: 0.9 * v.to(dt).double() for n, v in val.items()}
    d = {n: t.double() for n, t in w.items()}
    u = oracle.causal_conv(z["x"] + d["x.b"], d["conv"]) + d["conv.b"]
    s, S = oracle.gated_recurrence(u, oracle.sigmoid(oracle.block_linear(u, d["ra"], d["ra.b"])),
                                   oracle.sigmoid(oracle.block_linear(u, d["ri"], d["ri.b"])), d["lam"])
    want = s * oracle.gelu_tanh(z["y"] + d["y.b"])
    for cuts in ([T], [1] * T, [2] * 69 + [1], [64, 1, 63, 2, 9], [1, 65, 73], [3, 1, 1, 130, 4]):
        got, run, seq = run_core(blk, proj, cuts, kind)
        got = got[:, blk._out_columns()]
        tol = 2e-4 if dt == torch.float32 else 0.03
        assert (got - want).abs().max() < tol * float(want.abs().max()), cuts[:4]
        assert (run[1][seq.slot].cpu().double()[blk.geo.columns()] - S).abs().max() < (1e-4 if dt == torch.float32 else 0.02) * float(S.abs().max())


@pytest.mark.parametrize("kind", KINDS)
def test_rglru_starts_before_the_bias(kind):
    """Before the first token the convolution sees zeros, not the projection's bias; later it sees earlier inputs with their bias."""
    W, K = 16, 4
    blk = RGLRU(32, W, 1, K, getattr(torch, kind[1]), kind[0])
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    w["x.b"] += 1.0
    w["y.b"] += 3.0
    w["conv"] += torch.tensor([8.0, 4.0, 2.0, 1.0])
    w["lam"] += 20.0                                         # a is nearly 0 for r = 1: the state is i u
    w["ra.b"] += 20.0
    w["ri.b"] += 20.0
    blk.load(w)
    proj = packed(blk, 5, {"x": torch.zeros(5, W), "y": torch.zeros(5, W)}, kind)
    y = float(oracle.gelu_tanh(torch.tensor(3.0)))
    for cuts in ([5], [1] * 5, [2, 3], [3, 1, 1]):
        got, _, _ = run_core(blk, proj, cuts, kind)
        assert (got[:, 0] - y * torch.tensor([1.0, 3.0, 7.0, 15.0, 15.0])).abs().max() < (1e-4 if kind[1] == "float32" else 0.3), cuts


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
def test_mixed_batches_equal_each_alone(kind, graph):
    """Portions beside single tokens, requests that pause, end and give their pages and slot to others."""
    name = "odd"
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
    """Across spans, chunks, key tiles and splits: a prompt of 300 tokens in unequal portions, then decoding."""
    name = "plain"
    toks = tokens_for(CONFIGS[name], 420)
    want = reference(name, toks)
    eng = engine_for(name, kind, blocks=54)
    check(feed(eng, eng.open(), toks, [270, 30] + [1] * 120), want, kind)
    eng = engine_for(name, kind, blocks=54)
    check(feed(eng, eng.open(), toks, [5, 65, 256, 94]), want, kind)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["latent", "state"])
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
    cfg = polosun.preset("tiny", torch.float32)
    m = HybridModel(cfg, init_std=0.1, seed=3)
    p = tokens_for({"vocab": cfg.vocab_size}, 6)
    gen = GenerateConfig(max_new_tokens=8, do_sample=True, seed=11)
    out = m.generate(p, gen)
    assert len(out) == 14 and out == m.generate(p, gen)
    assert polosun.preset("small", torch.bfloat16).vocab_size == 4096
    with pytest.raises(ValueError, match="preset"):
        polosun.preset("huge", torch.float32)


# ---------------------------------------------------------------------------------------- files, registry, replay
def write_model(folder, name):
    from tesseract_b200.io.safetensors import save_file
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(CONFIGS[name]))
    save_file(weights_of(name), str(folder / "model.safetensors"), {})


@pytest.mark.parametrize("name", ["odd", "wide"])
def test_registry_files_and_round_trip(tmp_path, name):
    write_model(tmp_path / "m", name)
    m = load_pretrained(str(tmp_path / "m"), torch.float32, "cpu")
    assert isinstance(m, HybridModel) and m.config.architecture == "Polosun"
    arch = resolve(CONFIGS[name])
    from tesseract_b200.build import GROUPS
    assert arch.name == "Polosun" and arch.kernels in GROUPS
    assert polosun.config_to_dict(m.config) == CONFIGS[name]
    for k, t in m.state_tensors().items():
        assert torch.equal(t.to(torch.bfloat16), weights_of(name)[k]), k
    m.save_safetensors(str(tmp_path / "copy.safetensors"))
    again = HybridModel(m.config)
    assert again.load_safetensors(str(tmp_path / "copy.safetensors")) == []
    assert sum(t.numel() for t in m.parameters()) >= sum(t.numel() for t in weights_of(name).values())
    sd = dict(weights_of(name))
    for k in ("embed", "head", "l0.dwa", "l1.norm1", "l0.norm2", "final.norm", "l1.mix.dkv.norm" if name == "odd" else "l0.mix.uk", "l0.mlp.up"):
        with pytest.raises(KeyError, match="missing"):
            m.load_tensors({n: t for n, t in sd.items() if n != k})
    sd["l1.mix.o"] = sd["l1.mix.o"][:, 1:]
    with pytest.raises(ValueError, match="l1.mix"):
        m.load_tensors(sd)


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="ring"), "mixer"), (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"), (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), "rotary"), (lambda c: c["layers"][1]["mixer"].update(rot_dim=5), "rotary")])
def test_config_errors(change, what):
    c = json.loads(json.dumps(CONFIGS["odd"]))
    change(c)
    with pytest.raises(ValueError, match=what):
        polosun.config_from_dict(c)


def test_size_errors():
    r = Rotary(8, 1e4)
    for bad in (lambda: RetentionGeometry(2, 6, 8, r), lambda: RetentionGeometry(1, 264, 8, r), lambda: LatentGeometry(1, 8, 8, 8, 1020, r),
                lambda: LatentGeometry(1, 8, 6, 8, 16, r), lambda: RGLRUGeometry(10, 3, 2), lambda: log2_decays([1.5]),
                lambda: Retention(8, 2, 8, 8, (0.5,), r, 1e-5, torch.float32, "cpu")):
        with pytest.raises(ValueError):
            bad()
    att = AttentionSpec(1, 1, 8, 8, 1.0, 4)
    for kw in (dict(layers=[LayerSpec(att, SiluGLUSpec(8))], form="parallel"), dict(layers=[LayerSpec(att)], form="stacked"),
               dict(layers=[LayerSpec(att)], depth_average=True)):
        with pytest.raises(ValueError):
            HybridModel(HybridConfig(8, 8, **kw))


@pytest.mark.parametrize("kind", KINDS)
def test_mixers_also_run_in_sandwich_layers(kind):
    """The same mixers and the SiLU feed-forward between Dynamic Tanh norms, tied output: prompts against decoding."""
    src = polosun.config_from_dict(CONFIGS["plain"], getattr(torch, kind[1]))
    layers = [LayerSpec(s.mixer, s.mlp if i % 2 else GLUSpec(24, 2.0)) for i, s in enumerate(src.layers)]
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
    before = [[t.clone() for t in r] for r in eng.cache.runs]
    got = eng.execute([(s, t[11:]) for s, t in zip(seqs, toks)], [[0]] * 3)
    assert 4 in eng._graphs
    for r, b in zip(eng.cache.runs, before):
        for now, was in zip(r, b):
            rows = keep.get(now.shape[0], slice(None))          # (the angles do not change either)
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

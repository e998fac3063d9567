"""Tonilix (delta rule with decays per channel, attention with growing queries beside gated linear attention, mixtures of squared-ReLU
experts, pre-norms in parts, layer scales, a token shift, a sinusoid) against the plain statements of ``tonilix_oracle``: every mechanism
alone, prompts, portions, batches, decoding, reuse of pages and slots, and generation through the framework's entry points. The same
tests run on the CPU and, marked ``gpu``, on the kernels."""
import io
import json
import math

import numpy as np
import pytest
import torch

import tonilix_oracle as oracle
from tesseract_b200 import ops
from tesseract_b200.models import GenerateConfig, load_pretrained, tonilix
from tesseract_b200.models.hybrid import (Choice, DeltaSpec, ExpertSpec, GatedLinearSpec, GeluGLUSpec, HybridConfig, HybridModel, LayerSpec,
                                          ShapedAttentionSpec, SideBySideSpec)
from tesseract_b200.models.registry import resolve
from tesseract_b200.models.scheduler import ContinuousBatchingScheduler, EngineConfig
from tesseract_b200.nn.hybrid import ExpertMLP, GatedDelta, GatedLinear, ShapedAttention
from tesseract_b200.nn.ragged import HybridCache, HybridSequence, RaggedBatch
from tesseract_b200.ops.delta import DeltaGeometry
from tesseract_b200.ops.moe import Mixed, choose_experts_torch, relu2_experts, router_logits
from tesseract_b200.ops.pre_norm import Moved, Shift, pre_norm_step, sinusoid_frequencies
from tesseract_b200.ops.ragged import ScoreForm
from tesseract_b200.ops.timemix import GatedLinearGeometry
from tesseract_b200.serving import HybridEngine, make_engine

KINDS = [("cpu", "float32"), ("cpu", "bfloat16"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu),
         pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]
# relative error of a row of logits
TOL = {torch.float32: 2e-4, torch.bfloat16: 0.2}
MEAN_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.03}


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def moe(ff, experts, top, count=1, keep=1, scale=1.3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def delta(heads, kv, dim, vdim, conv, ra, rg, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": ra,
                                               "gate_rank": rg}, "mlp": mlp}


def pair(heads, kv, dim, vdim, lin_heads, lin_dim, lin_vdim, rank, tau=5.0, temp=(0.4, 7), scale=0.3, scales=(0.9, 0.6), mlp=None):
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                                                   "q_temp": {"coef": temp[0], "every": temp[1]}},
                                          "right": {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "tau": tau, "rank": rank},
                                          "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def conf(vocab, width, parts, layers, eps=1e-5):
    return {"architecture": "Tonilix", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": parts}, "layers": layers}


CONFIGS = {
    # sizes that are multiples of nothing, layers without a feed-forward, first and last ones of either kind, groups of one expert
    "odd": conf(53, 42, 3, [pair(6, 3, 10, 7, 3, 11, 5, 3, mlp=moe(13, 6, 2, 3, 2)), delta(6, 2, 9, 7, 4, 5, 3), delta(3, 3, 10, 13, 1, 7, 20, dense(31)),
                            pair(4, 4, 6, 9, 2, 5, 21, 17, tau=1.0, temp=(0.7, 1)), delta(2, 1, 21, 6, 6, 2, 2, moe(9, 5, 3, 5, 4)),
                            pair(5, 1, 7, 7, 1, 34, 3, 4, tau=16.0, mlp=dense(9))], 0.05),
    # sizes that the tensor-core kernels take; value heads that share key heads
    "plain": conf(130, 96, 2, [delta(4, 2, 64, 32, 3, 16, 24, moe(48, 12, 3, 3, 2)), pair(4, 2, 64, 64, 3, 32, 48, 16, scale=0.1, mlp=dense(72)),
                               delta(2, 2, 32, 64, 4, 8, 8, moe(32, 8, 2, 2, 1, scale=2.0)), pair(4, 1, 40, 64, 2, 64, 64, 8, tau=16.0, temp=(0.3, 64),
                               scale=0.1, mlp=moe(64, 16, 4, 4, 2))], 1e-6),
    # heads of 128 and heads and ranks that the fast kernels do not take
    "wide": conf(64, 128, 4, [delta(2, 1, 128, 128, 2, 40, 70, moe(96, 4, 1)), pair(2, 1, 128, 100, 2, 128, 80, 20, scale=0.1, mlp=moe(40, 70, 5, 7, 3)),
                              delta(1, 1, 200, 150, 8, 130, 16), pair(1, 1, 150, 200, 1, 150, 140, 70, scale=0.07, mlp=dense(64))]),
    # one kind each
    "delta": conf(40, 48, 1, [delta(4, 2, 16, 8, 3, 4, 4, dense(24)), delta(2, 2, 24, 8, 2, 9, 9)], 1e-4),
    "pair": conf(33, 32, 4, [pair(4, 1, 16, 8, 2, 16, 8, 4, mlp=dense(24)), pair(2, 1, 8, 16, 4, 8, 24, 3)], 0.05),
    "experts": conf(40, 48, 2, [delta(2, 2, 16, 16, 2, 4, 4, moe(24, 8, 2, 4, 2)), pair(2, 2, 16, 16, 2, 16, 16, 4, mlp=moe(16, 9, 4, 3, 2, scale=0.7))]),
}


def make_weights(config, seed=0):
    """bf16 tensors for every name the model has, sized so that no mechanism fades."""
    g = torch.Generator().manual_seed(seed)
    model = HybridModel(tonilix.config_from_dict(config))

    def draw(name, shape):
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last == "shift":
            return 0.2 + 0.6 * torch.rand(shape, generator=g)
        if last in ("ls1", "ls2"):
            return 0.5 + 0.3 * r
        if last == "A_log":
            return 0.7 * r - 1.0
        if last == "dt_bias":
            return 1.2 * r - 2.5
        if last == "correction":
            return 0.3 * r - 0.6                      # (choice scores of either sign)
        if last == "conv":
            return 0.6 * r
        if last == "b" and len(shape) == 1:
            return (2.0 if name.endswith("a2.b") else 0.4) * r
        if "norm" in last:
            return 0.3 * r + 1.0
        if name == "embed":
            return 0.7 * r
        return r * ((3.0 if last == "router" else 1.5) / math.sqrt(shape[-1]))
    w = {n: draw(n, s) for n, s in model.logical_shapes().items()}
    for n in list(w):
        if n.endswith("right.q"):      # the read-out over its own size has the sign of q . k: keep that away from zero
            w[n] = 0.8 * w[n[:-1] + "k"] + 0.6 * w[n]
    return {n: t.to(torch.bfloat16) for n, t in w.items()}


def make_model(config, weights, kind):
    m = HybridModel(tonilix.config_from_dict(config, getattr(torch, kind[1])), device=kind[0])
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


def reference(name, kind, toks):
    key = (name, kind[1], tuple(toks))
    if key not in _reference:
        _reference[key] = oracle.run_model(CONFIGS[name], weights_of(name, kind), toks)
    return _reference[key]


def weights_of(name, kind=("cpu", "float32")):
    """In bf16 the corrections decide which experts are taken: a close call is another expert, and that another result. What routing
    does otherwise is for the runs in fp32 and the tests of the choice alone."""
    key = (name, kind[1])
    if key not in _weights:
        w = make_weights(CONFIGS[name], seed=len(name))
        if kind[1] == "bfloat16":
            w = {n: 40.0 * t if n.endswith("correction") else t for n, t in w.items()}
        _weights[key] = w
    return _weights[key]


def engine_for(name, kind, blocks=64, block=8, batch=4, **kw):
    m = make_model(CONFIGS[name], weights_of(name, kind), kind)
    return HybridEngine(m, EngineConfig(block_size=block, num_blocks=blocks, max_seq_len=blocks * block, max_batch_size=batch), **kw)


def feed(eng, seq, toks, cuts):
    """Runs ``toks`` through one sequence in portions; logits of every token."""
    out, at = [], 0
    for n in cuts:
        out.append(eng.execute([(seq, toks[at:at + n])], [list(range(n))]))
        at += n
    assert at == len(toks)
    return torch.cat([o.float().cpu() for o in out])


# ---------------------------------------------------------------------------------------- the residual step
class Rows:
    """A ragged batch of one cache: (positions before, tokens) of every sequence, on slots that are not the first."""

    def __init__(self, kind, W, parts, vocab=19, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.cache = HybridCache([], 64, 8, 6, 512, getattr(torch, kind[1]), kind[0])
        self.cache.slot_allocator.allocate()
        C = (W + 15) // 16 * 16
        self.last = torch.randn(6, 1, C, generator=g).to(kind[0], getattr(torch, kind[1]))
        self.toks = {}
        self.g, self.vocab = g, vocab

    def batch(self, entries):
        toks = [(s, torch.randint(0, self.vocab, (n,), generator=self.g).tolist()) for s, n in entries]
        return RaggedBatch(self.cache, toks)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("W,parts,cols", [(40, 2, 48), (37, 1, 48), (42, 3, 48), (42, 21, 48), (256, 4, 256), (1030, 5, 1040), (2304, 2, 2304), (3000, 1, 3008),
                                          (12288, 3, 12288)])
def test_pre_norm_step_in_every_form(kind, W, parts, cols):
    dev, dt = kind[0], getattr(torch, kind[1])
    r = Rows(kind, W, parts, seed=W)
    g, eps = r.g, 1e-2
    rnd = lambda *s: torch.randn(*s, generator=g)   # noqa: E731
    vec = lambda off=0.0, by=0.3: (off + by * rnd(W)).to(dev)   # noqa: E731
    a, b = HybridSequence(r.cache), HybridSequence(r.cache)
    r.batch([(a, 300), (b, 3)]).commit()                       # (a is far in)
    batch = r.batch([(b, 5), (a, 1)])
    T = batch.rows
    pos = [300, 3, 4, 5, 6, 7]                                  # rows: the single token first
    table = torch.zeros(r.vocab, cols, dtype=dt)
    table[:, :W] = rnd(r.vocab, W)
    gain, egain = vec(1.0), vec(1.0)
    form = dict(out_cols=cols, out_dtype=dt)
    htol = 3e-5 if dt == torch.float32 else 0.05
    f64 = lambda t: t.double().cpu()   # noqa: E731
    freq = sinusoid_frequencies(W).to(dev)
    for f, e in ((None, None), (freq, None), (None, egain), (freq, egain)):
        x, h, moved = pre_norm_step(batch, W, gain, parts, eps, table=table.to(dev), freq=f, embed_gain=e, **form)
        want = table[batch.tokens.long().cpu(), :W].double()
        if f is not None:
            want = want + oracle.sinusoid(pos, W)
        if e is not None:
            want = oracle.part_rms_norm(want, f64(egain), parts, eps)
        assert moved is None and (f64(x) - want).abs().max() < 3e-6
        assert (f64(h[:, :W]) - oracle.part_rms_norm(want, f64(gain), parts, eps)).abs().max() < htol and float(h[:, W:].abs().sum()) == 0.0
    x0, y, bias, scale = rnd(T, W), (0.4 * rnd(T, cols)).to(dt), vec(by=0.2), vec(0.7)
    for bb, ss in ((None, None), (bias, None), (None, scale), (bias, scale)):
        xd = x0.to(dev)
        x, h, _ = pre_norm_step(batch, W, gain, parts, eps, xd, y.to(dev), bb, ss, **form)
        z = y[:, :W].double() + (f64(bias) if bb is not None else 0.0)
        want = x0.double() + z * (f64(scale) if ss is not None else 1.0)
        assert torch.equal(xd.cpu(), x0) and (f64(x) - want).abs().max() < 2e-6       # the residual stays in 32-bit whatever the type
        assert (f64(h[:, :W]) - oracle.part_rms_norm(want, f64(gain), parts, eps)).abs().max() < htol
    top = 3
    mixed = Mixed((0.4 * rnd(11, cols)).to(dt).to(dev), torch.randint(0, 11, (T, top), generator=g, dtype=torch.int32).to(dev),
                  torch.rand(T, top, generator=g).to(dev))
    x, h, _ = pre_norm_step(batch, W, gain, parts, eps, x0.to(dev), mixed, None, scale, **form)
    z = sum(f64(mixed.rows)[f64(mixed.pos[:, j]).long()] * f64(mixed.weight[:, j])[:, None] for j in range(top))[:, :W]
    assert (f64(x) - (x0.double() + z * f64(scale))).abs().max() < 3e-6


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("W,parts", [(40, 2), (37, 1), (1536, 3)])
def test_token_shift_across_rows_steps_and_slots(kind, W, parts):
    """Four sequences in portions beside single tokens: every row meets the one of the token before, whichever step or launch brought
    it; first tokens meet zeros on slots that hold something. The launches in between move the portions' last rows."""
    dev, dt = kind[0], getattr(torch, kind[1])
    r = Rows(kind, W, parts, seed=W)
    rnd = lambda *s: torch.randn(*s, generator=r.g)   # noqa: E731
    cols = r.last.shape[2]
    gain, mu, eps = (1 + 0.3 * rnd(W)).to(dev), torch.nn.functional.pad(rnd(W), (0, cols - W)).to(dev), 1e-3
    big = 2100 if dev == "cuda" and W == 40 else 20           # (more rows than a launch takes one by one)
    r.cache = HybridCache([], 800, 8, 6, 6000, dt, dev)
    r.cache.slot_allocator.allocate()
    seqs = [HybridSequence(r.cache) for _ in range(4)]
    plan = [[(0, 5), (1, 1)], [(1, 1), (0, 1), (2, 2)], [(2, 9), (0, big), (1, 1), (3, 1)], [(0, 1), (1, 3), (2, 17), (3, 2)], [(0, 1), (1, 1), (2, 1)]]
    moved, stream = None, {i: rnd(sum(dict(p).get(i, 0) for p in plan), W) for i in range(4)}
    want = {i: oracle.shifted_mix(oracle.part_rms_norm(s.double(), gain.double().cpu(), parts, eps), mu[:W].double().cpu()) for i, s in stream.items()}
    at = dict.fromkeys(stream, 0)
    for p in plan:
        batch = RaggedBatch(r.cache, [(seqs[i], [0] * n) for i, n in p])
        x = torch.empty(batch.rows, W)
        for e, (i, n) in enumerate(p):
            x[batch.row_of[e]:batch.row_of[e] + n] = stream[i][at[i]:at[i] + n]
        _, h, moved = pre_norm_step(batch, W, gain, parts, eps, x.to(dev), shift=Shift(mu, r.last), out_cols=cols, out_dtype=dt)
        if moved is not None:
            assert isinstance(moved, Moved)
            _, _, none = pre_norm_step(batch, W, gain, parts, eps, x.to(dev), moved=moved, out_cols=cols, out_dtype=dt)
            assert none is None
        for e, (i, n) in enumerate(p):
            got = h[batch.row_of[e]:batch.row_of[e] + n, :W].double().cpu()
            assert float(h[:, W:].abs().sum()) == 0.0
            assert (got - want[i][at[i]:at[i] + n]).abs().max() < (2e-5 if dt == torch.float32 else 0.1), (p, i)
            at[i] += n
        batch.commit()


# ---------------------------------------------------------------------------------------- mixers alone
def packed(block, T, values, kind):
    """The block's packed projection rows with the given logical values."""
    p = torch.zeros(T, block.cols)
    places = block._rows().items() if hasattr(block, "_rows") else ((n, at + torch.arange(k)) for n, at, k in block._sections())
    for name, rows in places:
        p[:, rows] = values[name].reshape(T, -1).float()
    return p.to(getattr(torch, kind[1])).to(kind[0])


def run_core(block, proj, cuts, kind, block_size=8):
    """Feeds rows of ``proj`` through a cache of one sequence whose slot and pages hold what an earlier one left."""
    T = proj.shape[0]
    n = (T + block_size - 1) // block_size
    cache = HybridCache([block.run_spec()], n + 3, block_size, 2, (n + 3) * block_size, block.dtype, kind[0])
    run = cache.runs[0]
    for t in run[:2]:
        if t is not None:
            t.copy_(torch.randn(t.shape).to(t.dtype))
    cache.allocator.allocate()                   # the sequence's pages and slot are not the pool's first
    cache.slot_allocator.allocate()
    seq, got, at = HybridSequence(cache), [], 0
    for n in cuts:
        b = RaggedBatch(cache, [(seq, [0] * n)], None, list(block.masks), 0, list(block.tiles))
        got.append(block.core(proj[at:at + n].contiguous(), run, b).float().cpu())
        b.commit()
        at += n
    assert at == T
    return torch.cat(got).double(), run, seq


def prompt_cuts(T, *edges):
    """Whole, token by token, pairs, and portions that end around the edges."""
    out = [[T], [1] * T, [2] * (T // 2) + [1] * (T % 2)]
    for e in edges:
        if 2 < e < T - 2:
            out += [[e, T - e], [e - 1, 2, T - e - 1], [e + 1] + [1] * min(7, T - e - 1) + ([T - e - 1 - min(7, T - e - 1)] if T - e - 8 > 0 else [])]
    return out


def delta_case(blk, T, kind, seed, loud=1.0):
    """(projection rows, logical values as rounded, weights) with decays from nearly 1 to nearly 0, different in every channel."""
    dt, gg = getattr(torch, kind[1]), blk.geo
    g = torch.Generator().manual_seed(seed)
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    for n in "qkv":
        w[n + ".conv"] = torch.randn(w[n + ".conv"].shape, generator=g) * 0.7
    w["A_log"] = torch.linspace(-1.0, 1.0, gg.heads)
    w["dt_bias"] = torch.linspace(-7.0, loud, gg.heads * gg.dim)[torch.randperm(gg.heads * gg.dim, generator=g)]
    w["norm"] = 1 + 0.3 * torch.randn(gg.vdim, generator=g)
    for n, k in (("a2", gg.decay_rank), ("g2", gg.gate_rank)):
        w[n] = torch.randn(w[n].shape, generator=g) * k ** -0.5
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    val = {n: torch.randn(T, k, generator=g) for n, _, k in blk._sections()}
    z = {n: t.to(dt).double() for n, t in val.items()}
    return packed(blk, T, val, kind), z, {n: t.double() for n, t in w.items()}


def delta_wanted(z, d, gg, eps):
    T, H, G = z["q"].shape[0], gg.heads, gg.kv_heads
    q, k, v = (oracle.silu(oracle.causal_conv(z[n], d[n + ".conv"])) for n in "qkv")
    q = (oracle.unit_vector(q.view(T, G, -1)) * gg.dim ** -0.5).repeat_interleave(H // G, dim=1)
    k = oracle.unit_vector(k.view(T, G, -1)).repeat_interleave(H // G, dim=1)
    decay = torch.exp(-torch.exp(d["A_log"])[:, None] * oracle.softplus((z["a1"] @ d["a2"].t() + d["dt_bias"]).view(T, H, -1)))
    o, S = oracle.channel_delta_recurrence(q, k, v.view(T, H, -1), decay, oracle.sigmoid(z["b"]))
    gate = oracle.sigmoid(z["g1"] @ d["g2"].t())
    return (oracle.over_rms(o, eps) * d["norm"]).reshape(T, -1) * gate, S, decay


DELTAS = [(3, 3, 10, 7, 4, 5, 3), (4, 2, 32, 16, 3, 16, 8), (6, 2, 64, 40, 2, 24, 24), (2, 1, 128, 128, 4, 20, 50), (2, 2, 200, 33, 1, 9, 8), (3, 1, 17, 130, 8, 2, 33),
          (8, 8, 64, 64, 4, 32, 32)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,G,D,E,K,ra,rg", DELTAS)
def test_channel_delta_alone(kind, H, G, D, E, K, ra, rg):
    dt, T, eps = getattr(torch, kind[1]), 75, 1e-2
    blk = GatedDelta(32, H, G, D, E, K, eps, dt, kind[0], ra, rg)
    proj, z, d = delta_case(blk, T, kind, D)
    want, S, decay = delta_wanted(z, d, blk.geo, eps)
    assert float(decay.min()) < 0.3 and float(decay.max()) > 0.99
    tol = 2e-4 if dt == torch.float32 else 0.03
    every = prompt_cuts(T, 4, 16, 33)
    for cuts in every[:2] + every[3:5] if kind[0] == "cpu" else every:
        got, run, seq = run_core(blk, proj, cuts, kind)
        err = (got[:, :H * E] - want).abs().max(1).values
        assert float(err.max()) < tol * max(1.0, float(want.abs().max())), (cuts[:4], int(err.argmax()))
        assert float(got[:, H * E:].abs().sum()) == 0.0
        state = run[1][seq.slot].cpu().double()[:, :, :E]
        assert (state - S).abs().max() < (1e-5 if dt == torch.float32 else 0.01) * max(1.0, float(S.abs().max())), cuts[:4]


@pytest.mark.parametrize("kind", KINDS)
def test_channel_delta_keeps_a_far_token_per_channel(kind):
    """One loud token far back and silence after it: every channel of the state holds it at the size that its own decay leaves."""
    dt, T, H, D, E = getattr(torch, kind[1]), 130, 2, 32, 8
    blk = GatedDelta(32, H, H, D, E, 2, 1e-6, dt, kind[0], 4, 4)
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    for n in "qkv":
        w[n + ".conv"][:, -1] = 1.0
    w["norm"] += 1.0
    w["dt_bias"] = torch.linspace(-8.0, -1.0, H * D)
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    decay = torch.exp(-oracle.softplus(w["dt_bias"].double())).view(H, D)
    v = float(torch.tensor(2.0).to(dt).double() / (1 + math.exp(-2.0)))
    for hot in (0, 3, 4, 15, 16, 63, 64):
        val = {n: torch.zeros(T, k) for n, _, k in blk._sections()}
        val["k"][hot], val["v"][hot], val["b"][:] = 2.0, 2.0, 20.0
        proj = packed(blk, T, val, kind)
        for cuts in ([T], [hot + 1, T - hot - 1], [T - 3, 1, 1, 1], [hot + 2, T - hot - 2]):
            _, run, seq = run_core(blk, proj, cuts, kind)
            st = run[1][seq.slot].cpu().double()[:, :, 3]
            want = D ** -0.5 * v * decay ** (T - 1 - hot)
            # (bf16 runs use the short form of the SiLU)
            assert ((st - want).abs() < (1e-4 if dt == torch.float32 else 1e-3) * want + 1e-12).all(), (hot, cuts)


def linear_case(blk, T, kind, seed, spread=6.0):
    dt, gg = getattr(torch, kind[1]), blk.geo
    g = torch.Generator().manual_seed(seed)
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    w["norm"] = 1 + 0.3 * torch.randn(gg.vdim, generator=g)
    w["a2"] = torch.randn(w["a2"].shape, generator=g) * gg.rank ** -0.5
    w["a2.b"] = torch.linspace(-spread, spread, gg.heads * gg.dim)[torch.randperm(gg.heads * gg.dim, generator=g)]
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    d = {n: t.double() for n, t in w.items()}
    val = {n: torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
    val["q"] = val["k"] + 0.5 * val["q"]
    z = {n: t.to(dt).double() for n, t in val.items()}
    decay = oracle.sigmoid(z["a1"] @ d["a2"].t() + d["a2.b"]) ** (1.0 / blk.w.tau)
    return packed(blk, T, val, kind), z, decay.view(T, gg.heads, gg.dim), d


def linear_wanted(z, decay, d, gg, eps, out_scale):
    T, H = decay.shape[:2]
    o, S = oracle.gated_linear_recurrence(z["q"].view(T, H, -1) * gg.dim ** -0.5, z["k"].view(T, H, -1), z["v"].view(T, H, -1), decay)
    return out_scale * (oracle.over_rms(o, eps) * d["norm"]).reshape(T, -1) * oracle.silu(z["g"]), S


LINEARS = [(3, 11, 5, 3), (4, 16, 16, 16), (2, 48, 64, 24), (3, 64, 20, 8), (2, 128, 100, 40), (2, 20, 128, 7), (1, 200, 33, 9), (2, 30, 140, 60)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("tau", [16.0, 1.0, 0.05])
@pytest.mark.parametrize("H,D,E,rank", LINEARS)
def test_gated_linear_alone(kind, tau, H, D, E, rank):
    """Decays from nearly 1 to (tau far below 1) nothing within a block."""
    dt, T, eps = getattr(torch, kind[1]), 141, 1e-2
    blk = GatedLinear(32, H, D, E, rank, tau, eps, dt, kind[0])
    blk.out_scale = 1.4
    proj, z, decay, d = linear_case(blk, T, kind, D)
    want, S = linear_wanted(z, decay, d, blk.geo, eps, 1.4)
    cols, tol = blk._out_columns(), 3e-4 if dt == torch.float32 else 0.03
    every = [[T], [64, 1, 63, 13], [1, 2, 15, 1, 16, 17, 89], [2] * 70 + [1], [128] + [1] * 13, [1] * T]
    for cuts in every[:2] if kind[0] == "cpu" else every:
        got, run, seq = run_core(blk, proj, cuts, kind)
        err = (got[:, cols] - want).abs().max(1).values
        assert float(err.max()) < tol * float(want.abs().max()), (cuts[:4], int(err.argmax()))
        rest = [i for i in range(got.shape[1]) if i not in set(cols.tolist())]
        assert float(got[:, rest].abs().sum()) == 0.0
        state = run[0][seq.slot].cpu().double()[:, :E, :D].transpose(1, 2)
        assert (state - S).abs().max() < (1e-4 if dt == torch.float32 else 0.01) * float(S.abs().max()), cuts[:4]


@pytest.mark.parametrize("kind", KINDS)
def test_gated_linear_keeps_a_far_token_per_channel(kind):
    dt, T, H, D, E, tau = getattr(torch, kind[1]), 150, 2, 32, 16, 8.0
    blk = GatedLinear(32, H, D, E, 4, tau, 1e-6, dt, kind[0])
    w = {n: torch.zeros(s) for n, s in blk.logical_shapes().items()}
    w["norm"] += 1.0
    w["a2.b"] = torch.linspace(-1.0, 6.0, H * D)
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    decay = (oracle.sigmoid(w["a2.b"].double()) ** (1 / tau)).view(H, D)
    for hot in (0, 15, 16, 63, 64, 127):
        val = {n: torch.zeros(T, len(r)) for n, r in blk._rows().items()}
        val["k"][hot], val["v"][hot] = 2.0, 3.0
        proj = packed(blk, T, val, kind)
        for cuts in ([T], [hot + 1, T - hot - 1], [T - 3, 1, 1, 1], [hot + 2, T - hot - 2]):
            _, run, seq = run_core(blk, proj, cuts, kind)
            st = run[0][seq.slot].cpu().double()[:, 5, :]
            want = 6.0 * decay ** (T - 1 - hot)
            assert ((st - want).abs() < 2e-4 * want + 1e-9).all(), (hot, cuts)


@pytest.mark.parametrize("kind", KINDS[1:])
@pytest.mark.parametrize("dim,vdim", [(32, 24), (128, 80), (20, 128)])
def test_long_portions_of_gated_linear_attention_are_walked_in_spans(kind, dim, vdim):
    """Portions longer than a span (and one just as long, one a token longer), from nothing and from what earlier ones left, beside
    a short one of another sequence."""
    dt, T, short, H = getattr(torch, kind[1]), 1085, 70, 2
    blk = GatedLinear(32, H, dim, vdim, 8, 16.0, 1e-2, dt, kind[0])
    proj, z, decay, d = linear_case(blk, T, kind, 5)
    want, S = linear_wanted(z, decay, d, blk.geo, 1e-2, 1.0)
    cols, tol = blk._out_columns(), (3e-4 if dt == torch.float32 else 0.03) * float(want.abs().max())
    for cuts in ([T], [512, 573], [513, 1, 571], [3, 1082]) if kind[0] == "cuda" else ([T],):
        got, run, seq = run_core(blk, proj, cuts, kind)
        err = (got[:, cols] - want).abs().max(1).values
        assert float(err.max()) < tol, (cuts, int(err.argmax()))
        state = run[0][seq.slot].cpu().double()[:, :vdim, :dim].transpose(1, 2)
        assert (state - S).abs().max() < (1e-4 if dt == torch.float32 else 0.01) * float(S.abs().max()), cuts
    cache = HybridCache([blk.run_spec()], 200, 8, 2, 1200, dt, kind[0])
    b = RaggedBatch(cache, [(HybridSequence(cache), [0] * short), (HybridSequence(cache), [0] * T)], None, list(blk.masks), 0, list(blk.tiles))
    got = blk.core(torch.cat([proj[:short], proj]), cache.runs[0], b).float().cpu().double()[:, cols]
    assert (got[:short] - want[:short]).abs().max() < tol and (got[short:] - want).abs().max() < tol


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,G,D,E,temp", [(4, 2, 12, 20, (0.4, 7.0)), (6, 3, 64, 40, (0.9, 1.0)), (2, 1, 128, 96, (0.3, 64.0)), (2, 1, 200, 130, (1.5, 50.0))])
def test_attention_with_growing_queries(kind, H, G, D, E, temp):
    """Queries at, before and after the edges of the temperature's steps, in prompts, portions and decoding."""
    dt, T = getattr(torch, kind[1]), 150
    blk = ShapedAttention(32, H, G, D, E, ScoreForm(D ** -0.5), 1e-6, dt, kind[0], bias=True, gate="element", q_temp=temp, out_bias=True)
    g = torch.Generator().manual_seed(D)
    w = {n: (torch.zeros(s) if len(s) == 2 else 0.5 * torch.randn(s, generator=g)).to(torch.bfloat16) for n, s in blk.logical_shapes().items()}
    blk.load(w)
    assert torch.equal(blk.out_bias.cpu(), w["o.b"].float())
    val = {n: torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
    proj = packed(blk, T, val, kind)
    z = {n: t.to(dt).double() for n, t in val.items()}
    q, k, v = ((z[n] + w[n + ".b"].double()).view(T, -1, d) for n, d in (("q", D), ("k", D), ("v", E)))
    loud = oracle.query_temperature(range(T), *temp)
    assert float(loud[-1]) > 1.2 and float(loud[0]) == 1.0 + temp[0] * math.log(math.floor(1 / temp[1]) + 1)
    want = oracle.attend(q * loud[:, None, None], k, v, D ** -0.5).reshape(T, -1) * oracle.sigmoid(z["g"])
    cuts = prompt_cuts(T, 64, 128)
    for c in cuts if kind[0] == "cuda" else cuts[:1] + cuts[3:5]:
        got, _, _ = run_core(blk, proj, c, kind)
        err = (got[:, blk._out_columns()] - want).abs().max(1).values
        assert float(err.max()) < (1e-4 if dt == torch.float32 else 0.04), (c[:4], int(err.argmax()))


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("D", [64, 100, 200])
def test_a_standing_out_key_is_found_from_everywhere(kind, D):
    """One key is made to win from its own token on: every later query returns its value, whatever page or portion it came with."""
    dt, T, H, G, E = getattr(torch, kind[1]), 290 if kind[0] == "cuda" else 80, 2, 1, 48
    blk = ShapedAttention(32, H, G, D, E, ScoreForm(1.0), 1e-6, dt, kind[0], bias=True, gate="element", q_temp=(0.2, 16.0), out_bias=True)
    blk.load({n: torch.zeros(s).to(torch.bfloat16) for n, s in blk.logical_shapes().items()})
    g = torch.Generator().manual_seed(7)
    for hot in (0, 7, 8, 63, 64, 127, 128, T - 1):
        if hot >= T:
            continue
        val = {n: 0.05 * torch.randn(T, len(r), generator=g) for n, r in blk._rows().items()}
        val["q"].view(T, H, D)[:, :, 1], val["k"].view(T, G, D)[hot, :, 1], val["v"][hot], val["g"][:] = 5.0, 8.0, 3.0, 20.0
        proj = packed(blk, T, val, kind)
        for cuts in ([T], [hot + 1, T - hot - 1] if hot + 1 < T else [T], [T - 20] + [1] * 20):
            got, _, _ = run_core(blk, proj, cuts, kind)
            o = got[:, blk._out_columns()]
            assert float((o[hot:] - 3.0).abs().max()) < 0.05 and (hot == 0 or float(o[:hot].abs().max()) < 0.5), (hot, cuts[:2])


# ---------------------------------------------------------------------------------------- feed-forwards alone
@pytest.mark.parametrize("kind", KINDS)
def test_gelu_unit(kind):
    dev, dt = kind[0], getattr(torch, kind[1])
    gu = torch.cat([torch.linspace(-30, 30, 64).expand(5, 64), torch.randn(5, 64)], dim=1).to(dt)
    got = ops.gelu_glu(gu.to(dev)).cpu().double()
    want = oracle.gelu_tanh(gu[:, :64].double()) * gu[:, 64:].double()
    assert ((got - want).abs() < (2e-6 if dt == torch.float32 else 0.01) * want.abs() + 1e-5).all()


CHOICES = [(16, 3, 2, 1), (6, 2, 3, 2), (5, 3, 5, 4), (12, 4, 3, 2), (8, 8, 1, 1), (70, 5, 7, 3), (256, 32, 16, 5), (9, 1, 1, 1), (64, 6, 8, 4)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("E,top,groups,keep", CHOICES)
@pytest.mark.parametrize("T", [1, 3, 70, 300])
def test_choice_of_experts(kind, E, top, groups, keep, T):
    """Experts and weights as stated, also where all choice scores are negative; experts without tokens; the sum over the chosen ones."""
    dev, dt, W, F = kind[0], getattr(torch, kind[1]), 40, 24
    if kind[0] == "cpu" and T == 300 and E > 16:
        pytest.skip("the same code as with fewer tokens")
    g = torch.Generator().manual_seed(E + T)
    c = Choice(E, top, groups, keep, 1.7)
    blk = ExpertMLP(W, F, c, dt, dev)
    w = {n: torch.randn(s, generator=g) / math.sqrt(s[-1]) for n, s in blk.logical_shapes().items()}
    w["correction"] = torch.randn(E, generator=g) * 0.4 - 0.8
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    blk.load(w)
    h = torch.randn(T, W, generator=g).to(dt)
    hp = torch.zeros(T, 48, dtype=dt)
    hp[:, :W] = h
    # logits that leave no close calls (the product itself is tested with whole models)
    logits = torch.zeros(T, (E + 7) // 8 * 8)
    for t in range(T):
        logits[t, :E] = torch.linspace(-4, 4, E)[torch.randperm(E, generator=g)] if E > 1 else 0.0
    corr = (w["correction"].double() * 0).float()
    corr += torch.linspace(-0.9, -0.95, E)          # (scores are at least 8 / E apart in the middle, the correction moves them little)
    s = oracle.sigmoid(logits[:, :E].double())
    parts = torch.stack([0.25 * logits, 0.75 * logits]) if T < 100 else logits[None]
    got = relu2_experts(hp.to(dev), parts.to(dev), corr.to(dev), c, blk.w_up, blk.w_down)
    d = {n: t.double() for n, t in w.items()}
    weights = got.weight.cpu().double()
    summed = got.sum().cpu().double()
    for t in range(0, T, max(1, T // 40)):
        ids = oracle.choose_experts(s[t], corr.double(), top, groups, keep)
        choice = sorted((float(s[t, e] + corr[e].double()) for e in range(E)), reverse=True)
        if min((a - b for a, b in zip(choice, choice[1:])), default=1.0) < 1e-6:
            continue
        total = sum(s[t, e] for e in ids) + 1e-20
        assert torch.allclose(weights[t].sort().values, torch.stack([s[t, e] / total * 1.7 for e in ids]).sort().values, atol=1e-6)
        want = sum(s[t, e] / total * 1.7 * (torch.clamp(h[t].double() @ d[f"e{e}.up"].t(), min=0) ** 2 @ d[f"e{e}.down"].t()) for e in ids)
        assert (summed[t] - want).abs().max() < (1e-4 if dt == torch.float32 else 0.03) * max(1.0, float(want.abs().max())), t


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("T,K,N", [(1, 16, 8), (5, 2048, 72), (40, 304, 16), (256, 784, 128), (300, 528, 8)])
def test_router_logits(kind, T, K, N):
    g, dt = torch.Generator().manual_seed(K), getattr(torch, kind[1])
    h, w = torch.randn(T, K, generator=g).to(dt), (torch.randn(N, K, generator=g) * K ** -0.5).to(dt)
    got = router_logits(h.to(kind[0]), w.to(kind[0]))
    assert got.dtype == torch.float32 and (got.sum(0).cpu().double() - h.double() @ w.double().t()).abs().max() < 2e-5      # in either type


def test_masked_experts_stay_out_although_all_scores_are_negative():
    """The best expert sits in the worse group: the groups' sums decide, and what is masked is below every negative score."""
    logits = torch.tensor([[4.0, -9.0, -9.0, -9.0, 1.0, 1.2, -9.0, -9.0]])
    corr = torch.full((8,), -2.0)
    idx, w = choose_experts_torch(logits, corr, Choice(8, 3, 2, 1, 1.0))
    assert sorted(idx[0].tolist())[:2] == [4, 5] and idx.min() >= 4
    idx, _ = choose_experts_torch(logits, corr, Choice(8, 3, 2, 2, 1.0))
    assert sorted(idx[0].tolist()) == [0, 4, 5]
    s = torch.sigmoid(logits[0].double())
    assert oracle.choose_experts(s, corr.double(), 3, 2, 1)[:2] == [5, 4] and oracle.choose_experts(s, corr.double(), 3, 2, 2) == [0, 5, 4]


@pytest.mark.parametrize("kind", KINDS[2:])
@pytest.mark.parametrize("T,E,W,F", [(700, 8, 96, 72), (1500, 5, 64, 64), (257, 64, 128, 48)])
def test_experts_of_long_prompts(kind, T, E, W, F):
    """As many rows as the grouped products and large tiles take, an expert that nearly all tokens choose, one that none does."""
    dt = getattr(torch, kind[1])
    g = torch.Generator().manual_seed(T)
    c = Choice(E, 2, 1, 1, 1.0)
    blk = ExpertMLP(W, F, c, dt, kind[0])
    w = {n: (torch.randn(s, generator=g) / math.sqrt(s[-1])).to(torch.bfloat16) for n, s in blk.logical_shapes().items()}
    blk.load(w)
    h = torch.zeros(T, blk.w_up.shape[2], dtype=dt)
    h[:, :W] = torch.randn(T, W, generator=g)
    logits = torch.randn(T, (E + 7) // 8 * 8, generator=g)
    logits[:, 0] += 6.0
    logits[:, E - 1] -= 12.0
    got = relu2_experts(h.to(kind[0]), logits[None].to(kind[0]), torch.zeros(E, device=kind[0]), c, blk.w_up, blk.w_down).sum().cpu().double()
    idx, weight = choose_experts_torch(logits[:, :E], torch.zeros(E), c)
    want = torch.zeros(T, W, dtype=torch.float64)
    for e in range(E):
        t, j = (idx == e).nonzero(as_tuple=True)
        y = torch.clamp(h[t, :W].double() @ w[f"e{e}.up"].double().t(), min=0) ** 2 @ w[f"e{e}.down"].double().t()
        want[t] += weight[t, j].double()[:, None] * y
    assert (got - want).abs().max() < (1e-4 if dt == torch.float32 else 0.03) * float(want.abs().max())


# ---------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer(kind, name):
    toks = tokens_for(CONFIGS[name], 41)
    trace = []
    want = oracle.run_model(CONFIGS[name], weights_of(name, kind), toks, trace=trace)
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
    want = reference(name, kind, toks)
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
    want = {i: reference(name, kind, t) for i, t in toks.items()}
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
    """Across blocks, tiles and splits: a prompt of 300 tokens in unequal portions, then decoding."""
    name = "plain"
    toks = tokens_for(CONFIGS[name], 420)
    want = reference(name, kind, toks)
    eng = engine_for(name, kind, blocks=54)
    check(feed(eng, eng.open(), toks, [270, 30] + [1] * 120), want, kind)
    eng = engine_for(name, kind, blocks=54)
    check(feed(eng, eng.open(), toks, [5, 65, 256, 94]), want, kind)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["delta", "pair", "experts"])
def test_far_and_first_tokens_reach_the_logits(kind, name):
    toks = tokens_for(CONFIGS[name], 30)
    other = [(toks[0] + 1) % CONFIGS[name]["vocab"]] + toks[1:]
    a, b = reference(name, kind, toks), reference(name, kind, other)
    assert float(row_error(a[-1:], b[-1:]).max()) > 3 * TOL[torch.float32]
    for t, w in ((toks, a), (other, b)):
        eng = engine_for(name, kind)
        check(feed(eng, eng.open(), t, [1, 2, 26, 1]), w, kind)


def test_wanted_rows_come_in_entry_order_and_nothing_is_kept_of_a_refused_step():
    kind = ("cpu", "float32")
    eng = engine_for("odd", kind, blocks=5, block=8, batch=2)
    ta, tb = tokens_for(CONFIGS["odd"], 12, 3), tokens_for(CONFIGS["odd"], 20, 4)
    a, b = eng.open(), eng.open()
    got = eng.execute([(a, ta), (b, tb[:1])], [[11, 2], [0]])
    check(got, torch.stack([reference("odd", kind, ta)[11], reference("odd", kind, ta)[2], reference("odd", kind, tb)[0]]), kind)
    assert eng.execute([(b, tb[1:3])], [[]]) is None
    with pytest.raises(RuntimeError, match="KV blocks"):
        eng.execute([(a, [1]), (b, tb[3:] + [0] * 20)], [[0], [0]])
    check(eng.execute([(b, tb[3:])], [range(17)]), reference("odd", kind, tb)[3:], kind)


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
    cfg = tonilix.preset("tiny", torch.float32)
    m = HybridModel(cfg, init_std=0.1, seed=3)
    p = tokens_for({"vocab": cfg.vocab_size}, 6)
    gen = GenerateConfig(max_new_tokens=8, do_sample=True, seed=11)
    out = m.generate(p, gen)
    assert len(out) == 14 and out == m.generate(p, gen)
    assert tonilix.preset("small", torch.bfloat16).vocab_size == 4096
    with pytest.raises(ValueError, match="preset"):
        tonilix.preset("huge", torch.float32)


# ---------------------------------------------------------------------------------------- files, registry, replay
def write_model(folder, name, config=None, kind=("cpu", "float32")):
    from tesseract_b200.io.safetensors import save_file
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config or CONFIGS[name]))
    save_file(weights_of(name, kind), str(folder / "model.safetensors"), {})


@pytest.mark.parametrize("name", ["odd", "wide"])
def test_registry_files_and_round_trip(tmp_path, name):
    write_model(tmp_path / "m", name)
    m = load_pretrained(str(tmp_path / "m"), torch.float32, "cpu")
    assert isinstance(m, HybridModel) and m.config.architecture == "Tonilix"
    arch = resolve(CONFIGS[name])
    from tesseract_b200.build import GROUPS
    assert arch.name == "Tonilix" and arch.kernels in GROUPS
    assert tonilix.config_to_dict(m.config) == CONFIGS[name]
    for k, t in m.state_tensors().items():
        assert torch.equal(t.to(torch.bfloat16), weights_of(name)[k]), k
    m.save_safetensors(str(tmp_path / "copy.safetensors"))
    again = HybridModel(m.config)
    assert again.load_safetensors(str(tmp_path / "copy.safetensors")) == []
    assert sum(t.numel() for t in m.parameters()) >= sum(t.numel() for t in weights_of(name).values())
    sd = dict(weights_of(name))
    for k in ("embed", "head", "embed.norm", "l0.norm1", "final.norm", "l0.ls1", "l1.shift", *(("l0.mix.left.o.b", "l0.mix.right.a2.b", "l1.mix.a2",
              "l1.mix.dt_bias", "l2.mix.g1", "l0.mlp.correction", "l0.mlp.e3.down", "l2.ls2") if name == "odd" else ())):
        with pytest.raises(KeyError, match="missing"):
            m.load_tensors({n: t for n, t in sd.items() if n != k})
    key = next(k for k in sd if k.startswith("l1.mix") and k.endswith(".o"))
    sd[key] = sd[key][:, 1:]
    with pytest.raises(ValueError, match="l1.mix"):
        m.load_tensors(sd)


def test_ranks_may_only_be_in_the_weights(tmp_path):
    config = json.loads(json.dumps(CONFIGS["odd"]))
    for l in config["layers"]:
        for m in (l["mixer"], l["mixer"].get("right", {})):
            for k in ("rank", "decay_rank", "gate_rank"):
                m.pop(k, None)
    write_model(tmp_path / "m", "odd", config)
    m = load_pretrained(str(tmp_path / "m"), torch.float32, "cpu")
    assert m.config == tonilix.config_from_dict(CONFIGS["odd"], torch.float32)
    toks = tokens_for(config, 20)
    check(m.forward(torch.tensor([toks]))[0], reference("odd", ("cpu", "float32"), toks), ("cpu", "float32"))


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="ring"), "mixer"), (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("q_temp"), "q_temp"), (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "kept"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "fewer")])
def test_config_errors(change, what):
    c = json.loads(json.dumps(CONFIGS["odd"]))
    change(c)
    with pytest.raises(ValueError, match=what):
        tonilix.config_from_dict(c)


def test_size_errors():
    for bad in (lambda: DeltaGeometry(1, 1, 8, 8, 2, 4, 0), lambda: DeltaGeometry(1, 1, 260, 8, 2, 4, 4), lambda: GatedLinearGeometry(1, 260, 8, 2),
                lambda: GatedLinearGeometry(1, 8, 8, 0), lambda: GatedLinear(8, 1, 8, 8, 2, 0.0, 1e-6, torch.float32, "cpu"),
                lambda: Choice(300, 2, 1, 1, 1.0), lambda: Choice(64, 40, 1, 1, 1.0)):
        with pytest.raises(ValueError):
            bad()
    d = DeltaSpec(1, 1, 8, 8, 2, 4, 4)
    experts = ExpertSpec(8, Choice(4, 2, 1, 1, 1.0))
    for kw in (dict(layers=[LayerSpec(d, experts)]), dict(layers=[LayerSpec(d)], norm_parts=2), dict(layers=[LayerSpec(d)], token_shift=True),
               dict(layers=[LayerSpec(d)], form="pre", norm_parts=3), dict(layers=[LayerSpec(d)], form="pre", norm_parts=0), dict(layers=[LayerSpec(d)], form="pre", embedding_scale=2.0)):
        with pytest.raises(ValueError):
            HybridModel(HybridConfig(8, 8, **kw))


@pytest.mark.parametrize("kind", KINDS)
def test_parts_of_the_design_run_in_other_forms(kind):
    """The mixers between Dynamic Tanh norms and in post-normed layers; pre-normed layers without scales, shift, sinusoid or norm of the
    embedding, of mixers without decays per channel: prompts against decoding."""
    dt = getattr(torch, kind[1])
    d, lin = DeltaSpec(4, 2, 32, 16, 3, 8, 8), GatedLinearSpec(2, 32, 24, 4.0, 8)
    att = ShapedAttentionSpec(2, 1, 64, 32, 0.1, window=20, norm="unit", q_temp=(0.3, 4.0))
    both = SideBySideSpec(ShapedAttentionSpec(2, 1, 64, 32, 0.1, bias=True, out_bias=True), lin, 0.5, 0.8)
    layers = [LayerSpec(d, GeluGLUSpec(24)), LayerSpec(lin, GeluGLUSpec(40)), LayerSpec(att)]
    configs = [HybridConfig(40, 48, layers + [LayerSpec(both)], dtype=dt), HybridConfig(40, 48, layers, dtype=dt, form="post"),
               HybridConfig(40, 48, layers + [LayerSpec(both, GeluGLUSpec(24)), LayerSpec(DeltaSpec(2, 2, 16, 16, 2))], dtype=dt, form="pre", norm_parts=2)]
    toks = tokens_for({"vocab": 40}, 70, 5)
    for c in configs:
        m = HybridModel(c, device=kind[0], init_std=0.2, seed=4)
        whole = m.forward(torch.tensor([toks]))[0].float().cpu()
        eng = HybridEngine(m, EngineConfig(block_size=8, num_blocks=16, max_seq_len=128, max_batch_size=2))
        check(feed(eng, eng.open(), toks, [40, 3, 7] + [1] * 20), whole, kind, c.form)


@pytest.mark.parametrize("kind", KINDS)
def test_trace_replay(kind, tmp_path):
    from tesseract_b200.serving.trace import make_replay, replay
    write_model(tmp_path / "m", "plain", kind=kind)
    c = CONFIGS["plain"]
    ta, tb = tokens_for(c, 25, 8), tokens_for(c, 30, 9)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ta[:20], "want": [0, 19]}, {"id": "y", "tokens": tb[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": tb[3:5], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": tb[5:6], "want": [0]}, {"id": "x", "tokens": ta[20:], "want": [4]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": tb[6:], "want": [23]}, {"id": "x", "tokens": tb[:1], "want": [0]}], "end": ["x", "y"]}]
    rep = make_replay(str(tmp_path / "m"), getattr(torch, kind[1]), torch.device(kind[0]), 64)
    said = []
    replay(rep, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(4)]
    ra, rb = reference("plain", kind, ta), reference("plain", kind, tb)
    for n, rows in {0: [ra[0], ra[19]], 2: [rb[5], ra[24]], 3: [rb[29], rb[0]]}.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(len(rows), -1))
        check(got, torch.stack(rows), kind, f"step {n}")
    assert rep.engine.allocated_blocks() == 0 and rep.live == {}


@pytest.mark.gpu
def test_padding_rows_of_a_captured_step_touch_nothing():
    """Three sequences decode in a bucket of four: the padding row leaves every page and slot alone."""
    kind = ("cuda", "bfloat16")
    eng = engine_for("plain", kind, blocks=24, batch=4)
    toks = [tokens_for(CONFIGS["plain"], 12, s) for s in range(3)]
    seqs = [eng.open() for _ in toks]
    eng.execute([(s, t[:11]) for s, t in zip(seqs, toks)], [[], [], []])
    eng.warm_graphs()
    used = {b for s in seqs for b in s.blocks}
    keep = {24: [b for b in range(24) if b not in used], 4: [3]}
    stores = [t for r in eng.cache.runs for t in eng.cache.tensors(r)]
    assert {t.shape[0] for t in stores} == {24, 4}
    before = [t.clone() for t in stores]
    got = eng.execute([(s, t[11:]) for s, t in zip(seqs, toks)], [[0]] * 3)
    assert 4 in eng._graphs
    for now, was in zip(stores, before):
        rows = keep[now.shape[0]]
        assert torch.equal(now[rows], was[rows])
    check(got, torch.stack([reference("plain", kind, t)[11] for t in toks]), kind)


@pytest.mark.gpu
def test_kernels_report_no_status():
    from tesseract_b200 import _native
    n0 = _native.launch_count()
    eng = engine_for("wide", ("cuda", "bfloat16"))
    feed(eng, eng.open(), tokens_for(CONFIGS["wide"], 20), [17, 1, 2])
    assert _native.launch_count() > n0
    assert _native.read_status(torch.cuda.current_stream().cuda_stream) == 0

"""Hybrid decoders (gated delta rule, chunked attention, Dynamic Tanh, looped layers, clamped GLU) against the plain
statements of ``hybrid_oracle``: every mechanism alone, prompts, portions, batches, decoding, reuse of pages and slots,
and generation through the framework's entry points. The same tests run on the CPU and, marked ``gpu``, on the kernels."""
import io
import json
import math

import numpy as np
import pytest
import torch

import hybrid_oracle as oracle
from tesseract_b200 import ops
from tesseract_b200.models import GenerateConfig, load_pretrained
from tesseract_b200.models import fozelix
from tesseract_b200.models.hybrid import HybridModel
from tesseract_b200.models.registry import resolve
from tesseract_b200.models.scheduler import ContinuousBatchingScheduler, EngineConfig
from tesseract_b200.nn.ragged import HybridCache, HybridSequence, PagedRun, RaggedBatch, StateRun, cut_segments
from tesseract_b200.ops.delta import DeltaGeometry, DeltaWeights
from tesseract_b200.ops.ragged import padded_head_dim
from tesseract_b200.serving import HybridEngine, make_engine

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
KINDS = [("cpu", "float32"), ("cpu", "bfloat16"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu),
         pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]
# relative error of a row of logits: bf16 rounding alone reaches 0.04 in single rows of the deepest configuration and
# 0.01 on average; a mechanism that is off by one token or factor shows as 0.3 and more
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.1}
MEAN_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.03}


def attn(heads, kv, dim, vdim, scale, size, ff=None, limit=1.0):
    mlp = {"kind": "dense", "ff": ff, "limit": limit} if ff else None
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": size}}, "mlp": mlp}


def delta(heads, kv, dim, vdim, conv, ff=None, limit=1.0):
    mlp = {"kind": "dense", "ff": ff, "limit": limit} if ff else None
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def conf(vocab, width, layers, loop=None, eps=1e-5, scale=1.0):
    c = {"architecture": "Fozelix", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
         "embedding": {"scale": scale}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # sizes that are multiples of nothing, a layer without feed-forward, a loop run three times in the middle
    "odd": conf(53, 42, [delta(4, 2, 10, 14, 4, 27, 0.8), attn(6, 2, 12, 20, 0.3, 7, 30, 1.1), delta(3, 1, 9, 5, 2),
                         attn(4, 4, 6, 10, 0.7, 11, 18, 0.6)], (1, 3, 3), 1e-3, 2.5),
    # no loop; 64-wide heads; as many key heads as heads
    "plain": conf(130, 96, [attn(3, 3, 64, 64, 0.2, 16, 72, 1.5), delta(3, 1, 32, 36, 3, 80, 0.9)], None, 1e-5, 4.0),
    # a loop over everything run once; sixteen heads on one key head; one tap; a head wider than 128
    "wide": conf(64, 128, [delta(2, 2, 130, 24, 1, 64, 2.0), attn(16, 1, 128, 96, 0.09, 33, 96, 0.7)], (0, 2, 1), 1e-6, 0.5),
    # query and key heads beyond 128, values narrow; a chunk of one token
    "tall": conf(40, 48, [attn(3, 1, 160, 32, 0.08, 5, 32, 1.0), attn(2, 1, 24, 40, 0.2, 1), delta(4, 1, 64, 132, 4, 40, 1.0)],
                 (1, 3, 2), 1e-5, 1.0),
    # recurrent only
    "delta": conf(33, 32, [delta(2, 1, 16, 16, 5, 24, 1.0), delta(2, 2, 20, 8, 8)], (0, 1, 2), 1e-4, 3.0),
}


def make_weights(config, seed=0):
    """bf16 tensors for every name the model has, sized so that no mechanism fades."""
    g = torch.Generator().manual_seed(seed)
    model = HybridModel(fozelix.config_from_dict(config))

    def draw(name, shape):
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last == "alpha":
            return 0.8 + 0.4 * torch.rand((), generator=g)
        if last == "A_log":
            return r * 0.7 - 1.0
        if last == "dt_bias":
            return r - 1.0
        if last == "conv":
            return r * 0.6
        if last == "b" and len(shape) == 1:
            return 0.3 * r
        if len(shape) == 1:
            return 1.0 + 0.3 * r
        if name == "loop.step":
            return 0.5 * r
        return r * (1.6 / math.sqrt(shape[1]))
    return {n: draw(n, s).to(torch.bfloat16) for n, s in model.logical_shapes().items()}


def make_model(config, weights, kind):
    device, dtype = kind[0], getattr(torch, kind[1])
    m = HybridModel(fozelix.config_from_dict(config, dtype), device=device)
    assert m.load_tensors(weights) == []
    return m


def tokens_for(config, n, seed=1):
    return np.random.default_rng(seed).integers(0, config["vocab"], n).tolist()


def row_error(got, want):
    got, want = got.double().cpu(), want.double()
    return ((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-6))


def check(got, want, kind, what=""):
    e = row_error(got, want)
    tol = TOL[getattr(torch, kind[1])]
    assert float(e.max()) < tol, f"{what}: worst row {int(e.argmax())} of {len(e)}: {float(e.max()):.2e} (limit {tol})"
    if len(e) >= 8:
        assert float(e.mean()) < MEAN_TOL[getattr(torch, kind[1])], f"{what}: mean {float(e.mean()):.2e}"


_reference = {}


def reference(name, toks):
    key = (name, tuple(toks))
    if key not in _reference:
        _reference[key] = oracle.run_model(CONFIGS[name], weights_of(name), toks)
    return _reference[key]


_weights = {}


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
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("W,cols", [(40, 48), (37, 48), (256, 256), (1030, 1040)])
def test_residual_step_in_every_form(kind, W, cols):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(W)
    T, V = 11, 19
    rnd = lambda *s: torch.randn(*s, generator=g)   # noqa: E731
    table = torch.zeros(V, cols, dtype=dt)
    table[:, :W] = rnd(V, W)
    toks = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    x0, y, yb, step = rnd(T, W), (2 * rnd(T, W)).to(dt), rnd(W), rnd(W)
    post, nxt = (0.7, rnd(W), rnd(W)), (1.3, rnd(W), rnd(W))
    d = lambda t: t.to(dev) if isinstance(t, torch.Tensor) else tuple(d(u) if isinstance(u, torch.Tensor) else u for u in t)  # noqa: E731
    e = oracle.embedding(toks.tolist(), table[:, :W].double(), 3.0)
    for embed, use_y, use_step, use_next in [("set", 0, 0, 1), ("set", 0, 1, 1), (None, 1, 0, 1), ("add", 1, 1, 1), (None, 1, 0, 0),
                                             ("add", 0, 1, 1)]:
        want = e.clone() if embed == "set" else x0.double()
        if use_y:
            want = want + oracle.dyn_tanh(y.double() + yb.double(), post[0], post[1].double(), post[2].double())
        if embed == "add":
            want = want + e
        if use_step:
            want = want + step.double()
        x = d(x0.clone())
        h = ops.dyn_tanh_residual(x, d(y) if use_y else None, d(yb) if use_y else None, d(post) if use_y else None,
                                  tokens=d(toks), table=d(table), scale=3.0, embed=embed, step=d(step) if use_step else None,
                                  next_norm=d(nxt) if use_next else None, out_cols=cols, out_dtype=dt)
        assert (x.cpu().double() - want).abs().max() < 2e-5          # the residual stays in 32-bit whatever the type
        if use_next:
            hw = oracle.dyn_tanh(want, nxt[0], nxt[1].double(), nxt[2].double())
            assert (h[:, :W].cpu().double() - hw).abs().max() < (2e-5 if dt == torch.float32 else 0.03)
            assert float(h[:, W:].abs().sum()) == 0.0
        else:
            assert h is None


@pytest.mark.parametrize("kind", KINDS)
def test_clamped_glu_cuts_gate_above_only_and_up_on_both_sides(kind):
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(0)
    F, limit = 48, 0.75
    gu, b = (3 * torch.randn(9, 2 * F, generator=g)).to(dt), torch.randn(2 * F, generator=g)
    z = gu.double() + b.double()
    want = oracle.clamped_glu(z[:, :F], z[:, F:], limit)
    got = ops.clamped_glu(gu.to(dev), b.to(dev), limit).cpu().double()
    assert (got - want).abs().max() < (1e-5 if dt == torch.float32 else 0.02)
    # a gate far below -limit still passes (it is not cut from below), one far above is cut; up likewise on both sides
    row = torch.tensor([[-2.0, 9.0, 0.5, 0.5] * 2 + [1.0, 1.0, -9.0, 9.0] * 2]).to(dt)
    want = oracle.clamped_glu(row[:, :8].double(), row[:, 8:].double(), limit)
    assert abs(float(want[0, 0])) > 0.1
    assert (ops.clamped_glu(row.to(dev), None, limit).cpu().double() - want).abs().max() < 0.01


def _attention_setup(kind, G, D_in, E_in, block, n_blocks, seqs=1):
    dev, dt = kind[0], getattr(torch, kind[1])
    D = padded_head_dim(D_in, E_in, dt)
    cache = HybridCache([PagedRun(G, D)], n_blocks, block, seqs, n_blocks * block, dt, dev)
    return cache, D


def _pack_qkv(q, k, v, D, kind):
    """[T, H, d], [T, G, d], [T, G, e] -> the padded packed rows."""
    T = q.shape[0]
    parts = []
    for t in (q, k, v):
        p = torch.zeros(T, t.shape[1], D)
        p[:, :, :t.shape[2]] = t
        parts.append(p.reshape(T, -1))
    return torch.cat(parts, 1).to(getattr(torch, kind[1])).to(kind[0])


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,G,D,E,chunk", [(4, 2, 64, 64, 24), (3, 3, 40, 20, 9), (8, 1, 128, 128, 40), (2, 1, 150, 70, 13)])
def test_one_standing_out_key_at_every_chunk_edge(kind, H, G, D, E, chunk):
    """One key is made to win wherever it is seen, and its value to be unmistakable: a query just inside its chunk returns
    that value, the first query of the next chunk must not -- in a prompt, in portions and in decoding."""
    dt = getattr(torch, kind[1])
    g = torch.Generator().manual_seed(chunk)
    T, block = 3 * chunk + 2, 8
    for hot in (0, chunk - 1, chunk, 2 * chunk - 1, 2 * chunk, T - 1):
        q = torch.randn(T, H, D, generator=g) * 0.1
        k = torch.randn(T, G, D, generator=g) * 0.1
        v = torch.randn(T, G, E, generator=g)
        q[:, :, 0], k[hot, :, 0], v[hot] = 6.0, 6.0, 7.0
        q, k, v = (t.to(dt).float() for t in (q, k, v))
        want = oracle.chunked_attention(q.double(), k.double(), v.double(), 0.5, chunk)
        seen = [i for i in range(hot, T) if i // chunk == hot // chunk]
        assert (want[seen] - 7.0).abs().max() < 0.1
        for cuts in ([T], [chunk - 1, 2, T - chunk - 1], [1] * T, [hot + 1, T - hot - 1] if hot + 1 < T else [T - 1, 1]):
            cache, Dp = _attention_setup(kind, G, D, E, block, (T + block - 1) // block + 2)
            seq = HybridSequence(cache)
            cache.allocator.allocate()           # the sequence's pages are not the pool's first
            qkv = _pack_qkv(q, k, v, Dp, kind)
            got, at = [], 0
            for n in cuts:
                b = RaggedBatch(cache, [(seq, [0] * n)], None, [chunk])
                kp, vp = cache.runs[0]
                o = ops.ragged_attention(qkv[at:at + n].contiguous(), None, kp, vp, b, H, G, 0.5, chunk)
                b.commit()
                got.append(o.view(n, H, Dp)[:, :, :E].float().cpu())
                at += n
            got = torch.cat(got).double()
            assert (got - want).abs().max() < (1e-4 if dt == torch.float32 else 0.06), (hot, cuts[:3])


@pytest.mark.parametrize("kind", KINDS)
def test_attention_bias_scale_and_unmasked_form(kind):
    """Biases enter before the scores, the scale is the caller's, and chunk 0 is plain causal attention."""
    dev, dt = kind[0], getattr(torch, kind[1])
    g = torch.Generator().manual_seed(5)
    H, G, D, T = 4, 2, 64, 45
    cache, Dp = _attention_setup(kind, G, D, D, 16, 6)
    z = torch.randn(T, (H + 2 * G) * D, generator=g).to(dt)
    b = torch.randn((H + 2 * G) * D, generator=g)
    zz = (z.double() + b.double()).view(T, H + 2 * G, D)
    want = oracle.chunked_attention(zz[:, :H], zz[:, H:H + G], zz[:, H + G:], 0.03, 10 ** 6)
    seq = HybridSequence(cache)
    got, at = [], 0
    for n in (30, 1, 14):
        batch = RaggedBatch(cache, [(seq, [0] * n)], None, [0])
        got.append(ops.ragged_attention(z[at:at + n].to(dev), b.to(dev), *cache.runs[0], batch, H, G, 0.03, 0))
        batch.commit()
        at += n
    got = torch.cat(got).view(T, H, D).cpu().double()
    assert (got - want).abs().max() < (1e-4 if dt == torch.float32 else 0.05)


def test_segments_cut_at_chunk_edges():
    s = cut_segments([(5, 9), (0, 2), (8, 8)], 4, lambda i, p: p + 100 * i)
    cu_q, cu_k, rows, dst, src = (h.tolist() for h in s.host)
    assert cu_q == [0, 3, 7, 9, 11, 15, 19]                    # 5..7 | 8..11 | 12..13, 0..1, 8..11 | 12..15
    assert cu_k == [0, 4, 8, 10, 12, 16, 20]                   # the first piece also sees position 4
    assert dst == [0] and src == [4] and rows == list(range(1, 20))
    assert (s.n, s.max_q, s.keys, s.n_gather) == (6, 4, 20, 1)
    assert cut_segments([(5, 9)], 0, lambda i, p: p).host[1].tolist() == [0, 14]
    assert cut_segments([(3, 1), (4, 4)], 1, lambda i, p: p).n == 5


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,G,D,E,K", [(4, 2, 16, 24, 3), (3, 1, 10, 7, 4), (2, 2, 128, 128, 2), (6, 3, 40, 33, 1), (2, 1, 200, 12, 8)])
def test_delta_rule_alone(kind, H, G, D, E, K):
    """Convolution, unit vectors, gates, recurrence and read-out against the token-by-token statement; in portions of every
    kind, with the state left in a slot that another sequence had used."""
    dev, dt = kind[0], getattr(torch, kind[1])
    geo = DeltaGeometry(G, H, D, E, K)
    g = torch.Generator().manual_seed(D)
    T, eps = 37, 1e-3
    proj = torch.zeros(T, geo.cols)
    sec = {"q": (0, G * D), "k": (geo.off_k, G * D), "v": (geo.off_v, H * E), "g": (geo.off_gate, H * E), "b": (geo.off_b, H),
           "a": (geo.off_a, H)}
    for o, n in sec.values():
        proj[:, o:o + n] = torch.randn(T, n, generator=g)
    proj = proj.to(dt)
    taps = {n: torch.randn(sec[n][1], K, generator=g) for n in "qkv"}
    conv = torch.zeros(K, geo.conv_cols)
    for n in "qkv":
        conv[:, sec[n][0]:sec[n][0] + sec[n][1]] = taps[n].t()
    a_log, dt_bias, norm = (torch.randn(n, generator=g) for n in (H, H, E))
    p = proj.double()
    part = lambda n: p[:, sec[n][0]:sec[n][0] + sec[n][1]]    # noqa: E731
    q, k, v = (oracle.silu(oracle.causal_conv(part(n), taps[n].double())) for n in "qkv")
    q, k = q.view(T, G, D), k.view(T, G, D)
    q, k = oracle.unit_vector(q) * D ** -0.5, oracle.unit_vector(k)
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    decay = torch.exp(-torch.exp(a_log.double()) * oracle.softplus(part("a") + dt_bias.double()))
    beta = 1 / (1 + torch.exp(-part("b")))
    o, S = oracle.delta_recurrence(q, k, v.view(T, H, E), decay, beta)
    want = oracle.gated_head_norm(o, part("g").view(T, H, E), norm.double(), eps).reshape(T, H * E)
    w = DeltaWeights(*(t.to(dev) for t in (conv, a_log, dt_bias, norm)), eps)
    for cuts in ([T], [1] * T, [2] * 18 + [1], [17, 1, 1, 16, 2], [1, 36]):
        cache = HybridCache([StateRun((H, D, geo.vdim_pad), (K - 1, geo.conv_cols))], 40, 1, 1, 40, dt, dev)
        cs, st = cache.runs[0]
        cs.fill_(3.0)
        st.fill_(-2.0)                            # what a sequence before left in the slot
        if geo.vdim_pad > E:
            st[..., E:] = 0
        seq, got, at = HybridSequence(cache), [], 0
        for n in cuts:
            b = RaggedBatch(cache, [(seq, [0] * n)], None, [])
            got.append(ops.gated_delta(proj[at:at + n].to(dev), geo, w, cs, st, b))
            b.commit()
            at += n
        got = torch.cat(got).cpu().double()
        tol = 2e-4 if dt == torch.float32 else 0.03 * float(want.abs().max())
        assert (got[:, :H * E] - want).abs().max() < tol, cuts[:4]
        assert float(got[:, H * E:].abs().sum()) == 0.0
        assert (st[0, :, :, :E].cpu().double() - S).abs().max() < 1e-4     # the state is 32-bit in both types


# ---------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer(kind, name):
    toks = tokens_for(CONFIGS[name], 41)
    trace = []
    want = oracle.run_model(CONFIGS[name], weights_of(name), toks, trace=trace)
    eng = engine_for(name, kind)
    seen = []
    seq = eng.open()
    b = eng.model.make_batch(eng.cache, [(seq, toks)], [range(41)])
    got = eng.model.forward_ragged(b, eng.cache, on_layer=lambda r, x: seen.append((r, x.cpu().double())))
    check(got, want, kind, "logits")
    assert [r for r, _ in seen] == list(range(len(trace))) == list(range(len(eng.model.runs)))
    for (r, x), t in zip(seen, trace):
        assert float(row_error(x, t).max()) < TOL[getattr(torch, kind[1])], f"residual after run {r}"
    plain = eng.execute([(eng.open(), toks)], [range(41)])       # without the hook: the fused form of the same step
    check(plain, want, kind, "fused")
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
def test_long_decoding_across_many_chunks(kind):
    name = "plain"
    toks = tokens_for(CONFIGS[name], 170)
    want = reference(name, toks)
    eng = engine_for(name, kind, blocks=24)
    check(feed(eng, eng.open(), toks, [5] + [1] * 165), want, kind)


@pytest.mark.parametrize("kind", KINDS)
def test_far_and_first_tokens_reach_the_logits(kind):
    """The state carries the first token to the end; a chunk's attention forgets everything before its edge."""
    name = "delta"
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
    got = eng.execute([(a, ta), (b, tb[:1])], [[11, 2], [0]])          # the single token's row is placed first in the batch
    want = torch.stack([reference("odd", ta)[11], reference("odd", ta)[2], reference("odd", tb)[0]])
    check(got, want, ("cpu", "float32"))
    assert eng.execute([(b, tb[1:3])], [[]]) is None
    with pytest.raises(RuntimeError, match="KV blocks"):
        eng.execute([(a, [1]), (b, tb[3:] + [0] * 20)], [[0], [0]])
    with pytest.raises(RuntimeError, match="slots"):
        eng.execute([(a, [1]), (eng.open(), [1])], [[0], [0]])
    with pytest.raises(ValueError, match="vocab"):
        eng.execute([(a, [CONFIGS["odd"]["vocab"]])], [[0]])
    check(eng.execute([(b, tb[3:])], [range(17)]), reference("odd", tb)[3:], ("cpu", "float32"))
    assert (a.length, b.length) == (12, 20)


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
        assert eng.allocated_blocks() == 0 and eng._promised == 0 and eng.metrics()["requests"] == len(prompts)
    # the per-request scheduler that also serves the framework's CPU and 32-bit models
    sch = ContinuousBatchingScheduler(m, EngineConfig(block_size=8, num_blocks=32, max_seq_len=48, max_batch_size=3))
    ids = [sch.add_request(p, gen) for p in prompts]
    sch.run()
    assert [sch.result(i) for i in ids] == want


def test_sampling_eos_and_limits():
    m = make_model(CONFIGS["plain"], weights_of("plain"), ("cpu", "float32"))
    p = tokens_for(CONFIGS["plain"], 6)
    cfg = GenerateConfig(max_new_tokens=8, do_sample=True, seed=11)
    out = m.generate(p, cfg)
    assert len(out) == 14 and out == m.generate(p, cfg)
    sch = ContinuousBatchingScheduler(m, EngineConfig(block_size=8, num_blocks=16, max_seq_len=32, max_batch_size=2))
    rid = sch.add_request(p, cfg)
    sch.run()
    assert sch.result(rid) == out                                  # same sampler, same logits, either scheduler
    first = m.generate(p, GenerateConfig(max_new_tokens=1))[-1]
    assert m.generate(p, GenerateConfig(max_new_tokens=8, eos_token_id=first)) == p + [first]
    assert m.generate(p, GenerateConfig(max_new_tokens=0)) == p
    with pytest.raises(ValueError):
        m.generate([], cfg)
    with pytest.raises(ValueError):
        m.generate(p, GenerateConfig(kv_int8=True))
    eng = make_engine(m, EngineConfig(block_size=8, num_blocks=2, max_seq_len=64, max_batch_size=2))
    with pytest.raises(ValueError, match="never fit"):
        eng.add_request(p, GenerateConfig(max_new_tokens=20))
    assert not eng.has_pending()


def test_grammar_constrained_generation():
    from tesseract_b200.models.structured import generate_structured
    m = make_model(CONFIGS["plain"], weights_of("plain"), ("cpu", "float32"))

    class Bytes:
        def decode(self, ids, skip_special_tokens=True):
            return bytes(ids).decode("latin-1")
    out = generate_structured(m, [49, 50], Bytes(), "[0-9]+", GenerateConfig(max_new_tokens=5))
    assert len(out) == 7 and all(48 <= t < 58 for t in out)


# ---------------------------------------------------------------------------------------- files, registry, replay
def write_model(folder, name):
    from tesseract_b200.io.safetensors import save_file
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(CONFIGS[name]))
    save_file(weights_of(name), str(folder / "model.safetensors"), {})


def test_registry_files_and_round_trip(tmp_path):
    write_model(tmp_path / "m", "tall")
    m = load_pretrained(str(tmp_path / "m"), torch.float32, "cpu")
    assert isinstance(m, HybridModel) and m.config.architecture == "Fozelix"
    assert fozelix.config_to_dict(m.config) == {**CONFIGS["tall"]}
    for k, t in m.state_tensors().items():
        assert torch.equal(t.to(torch.bfloat16), weights_of("tall")[k]), k
    m.save_safetensors(str(tmp_path / "copy.safetensors"))
    again = HybridModel(m.config)
    assert again.load_safetensors(str(tmp_path / "copy.safetensors")) == []
    assert resolve({"hidden_size": 8, "architectures": ["LlamaForCausalLM"]}).name == "Llama"
    for bad in ({}, {"architecture": "Other", "hidden_size": 8}):
        with pytest.raises(ValueError, match="no registered model"):
            resolve(bad)
    sd = dict(weights_of("tall"))
    sd["extra"] = torch.zeros(1)
    assert m.load_tensors(sd) == ["extra"]
    for k in ("embed", "loop.step", "l0.mix.q.b", "l1.norm1b.alpha", "l2.mix.v.conv", "l2.mlp.up.b", "final.norm"):
        with pytest.raises(KeyError, match="missing"):
            m.load_tensors({n: t for n, t in sd.items() if n != k})
    sd["l2.mix.o"] = sd["l2.mix.o"][:, 1:]
    with pytest.raises(ValueError, match="l2.mix"):
        m.load_tensors(sd)


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="ring"), "mixer"), (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["loop"].update(stop=9), "loop"), (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"), (lambda c: c.pop("width"), "width"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask")])
def test_config_errors(change, what):
    c = json.loads(json.dumps(CONFIGS["odd"]))
    change(c)
    with pytest.raises(ValueError, match=what):
        fozelix.config_from_dict(c)


def test_size_errors():
    with pytest.raises(ValueError):
        DeltaGeometry(2, 3, 8, 8, 2)
    with pytest.raises(ValueError):
        DeltaGeometry(1, 1, 257, 8, 2)
    with pytest.raises(ValueError):
        padded_head_dim(300, 8, torch.float32)


@pytest.mark.parametrize("kind", KINDS)
def test_trace_replay(kind, tmp_path):
    """Steps as JSON lines in, logits of the wanted places out; a request that ends makes room for the next."""
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
    assert not (tmp_path / "1.f32").exists()
    ra, rb = reference("odd", ta), reference("odd", tb)
    want = {0: [ra[0], ra[19]], 2: [rb[5], ra[24]], 3: [rb[29], rb[0]]}
    for n, rows in want.items():
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
    free = [b for b in range(24) if b not in used]
    before = [[t.clone() for t in r] for r in eng.cache.runs]
    got = eng.execute([(s, t[11:]) for s, t in zip(seqs, toks)], [[0]] * 3)
    assert 4 in eng._graphs
    for r, b in zip(eng.cache.runs, before):
        for now, was in zip(r, b):
            keep = free if now.shape[0] == 24 else [3]
            assert torch.equal(now[keep], was[keep])
    check(got, torch.stack([reference("plain", t)[11] for t in toks]), ("cuda", "bfloat16"))


@pytest.mark.gpu
def test_kernels_report_no_status():
    from tesseract_b200 import _native
    n0 = _native.launch_count()
    eng = engine_for("wide", ("cuda", "bfloat16"))
    feed(eng, eng.open(), tokens_for(CONFIGS["wide"], 20), [17, 1, 2])
    assert _native.launch_count() > n0
    assert _native.read_status(torch.cuda.current_stream().cuda_stream) == 0

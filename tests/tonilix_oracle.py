"""Plain statements of Tonilix's mechanisms, one function each, in the slowest readable form: one sequence at a time, in float64 by
default, sharing no code with the package. Mechanisms that other designs also have come from the other oracles."""
from __future__ import annotations

import math

import torch

from hybrid_oracle import causal_conv, linear, silu, softplus, unit_vector
from polosun_oracle import gelu_tanh, over_rms, sigmoid
from vobotar_oracle import attend, shifted_mix


def sinusoid(positions, width):
    """[T, width]: neighbours (2 i, 2 i + 1) hold sine and cosine of p / 10000^(2 i / width)."""
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for t, p in enumerate(positions):
        for c in range(width):
            a = p * 10000.0 ** (-2.0 * (c // 2) / width)
            out[t, c] = math.sin(a) if c % 2 == 0 else math.cos(a)
    return out


def part_rms_norm(x, weight, parts, eps):
    """Equal runs of neighbours, every one over its own root mean square; then a weight per channel."""
    T, W = x.shape
    return over_rms(x.view(T, parts, W // parts), eps).reshape(T, W) * weight


# ------------------------------------------------------------------------------------------ delta rule with channel decays
def channel_delta_recurrence(q, k, v, decay, beta, state=None):
    """q, k, decay [T, H, D], v [T, H, E], beta [T, H]; state [H, D, E]. Returns (o [T, H, E], state)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, :, None] * S
        seen = (S * k[t][:, :, None]).sum(1)
        u = beta[t][:, None] * (v[t] - seen)
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def channel_decay(h, w, heads):
    """exp(-exp(A_log) softplus(..)): [T, heads, dim]."""
    z = linear(linear(h, w["a1"]), w["a2"]) + w["dt_bias"]
    return torch.exp(-torch.exp(w["A_log"])[:, None] * softplus(z.view(h.shape[0], heads, -1)))


def channel_delta_mixer(h, w, m, eps):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(linear(h, w[n]), w[n + ".conv"])) for n in "qkv")
    q = (unit_vector(q.view(T, G, D)) * D ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit_vector(k.view(T, G, D)).repeat_interleave(H // G, dim=1)
    o, _ = channel_delta_recurrence(q, k, v.view(T, H, E), channel_decay(h, w, H), sigmoid(linear(h, w["b"])))
    gate = sigmoid(linear(linear(h, w["g1"]), w["g2"]))
    return linear((over_rms(o, eps) * w["norm"]).reshape(T, H * E) * gate, w["o"])


# ------------------------------------------------------------------------------------------ attention beside gated linear attention
def query_temperature(positions, coef, every):
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in positions], dtype=torch.float64)


def gated_attention(h, w, m):
    """Biases on all four projections, queries louder with their position, a gate per element."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w["q"], w["q.b"]).view(T, H, D)
    k = linear(h, w["k"], w["k.b"]).view(T, G, D)
    v = linear(h, w["v"], w["v.b"]).view(T, G, E)
    q = q * query_temperature(range(T), m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None]
    o = attend(q, k, v, m["scale"]).reshape(T, H * E) * sigmoid(linear(h, w["g"]))
    return linear(o, w["o"], w["o.b"])


def gated_linear_recurrence(q, k, v, decay, state=None):
    """q, k, decay [T, H, D], v [T, H, E]; state [H, D, E]. Returns (o [T, H, E], state)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def gated_linear_mixer(h, w, m, eps):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = linear(h, w["q"]).view(T, H, D) * D ** -0.5, linear(h, w["k"]).view(T, H, D)
    decay = sigmoid(linear(linear(h, w["a1"]), w["a2"], w["a2.b"])) ** (1.0 / m["tau"])
    o, _ = gated_linear_recurrence(q, k, linear(h, w["v"]).view(T, H, E), decay.view(T, H, D))
    o = (over_rms(o, eps) * w["norm"]).reshape(T, H * E)
    return linear(o * silu(linear(h, w["g"])), w["o"])


def parallel_mixer(h, w, m, eps):
    left, right = ({n[len(p):]: t for n, t in w.items() if n.startswith(p)} for p in ("left.", "right."))
    return m["left_scale"] * gated_attention(h, left, m["left"]) + m["right_scale"] * gated_linear_mixer(h, right, m["right"], eps)


# ------------------------------------------------------------------------------------------ feed-forwards
def gelu_feed_forward(h, w):
    return linear(gelu_tanh(linear(h, w["gate"])) * linear(h, w["up"]), w["down"])


def choose_experts(scores, correction, top, groups, keep):
    """One token's expert ids, by score + correction, from the groups whose two best sums are largest."""
    choice = [float(s) + float(c) for s, c in zip(scores, correction)]
    size = len(choice) // groups
    worth = [sum(sorted(choice[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -worth[g])[:keep]
    allowed = [e for e in range(len(choice)) if e // size in kept]
    return sorted(allowed, key=lambda e: -choice[e])[:top]


def mixture(h, w, m):
    r = m["router"]
    scores = sigmoid(linear(h, w["router"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose_experts(scores[t], w["correction"], r["top"], r["groups"]["count"], r["groups"]["keep"])
        total = sum(scores[t, e] for e in ids) + 1e-20
        for e in ids:
            y = linear(torch.clamp(linear(h[t], w[f"e{e}.up"]), min=0.0) ** 2, w[f"e{e}.down"])
            out[t] += scores[t, e] / total * r["scale"] * y
    return out


# ------------------------------------------------------------------------------------------ the model
def run_model(config, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one whole sequence. ``trace`` (a list) receives the residual after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps, parts = config["norm"]["eps"], config["norm"]["groups"]
    toks = torch.as_tensor(tokens, dtype=torch.long)

    def sub(prefix):
        return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}

    def norm(name, x):
        return part_rms_norm(x, W[name], parts, eps)

    x = norm("embed.norm", W["embed"][toks] + sinusoid(range(len(toks)), config["width"]).to(dtype))
    for i, spec in enumerate(config["layers"]):
        h = shifted_mix(norm(f"l{i}.norm1", x), W[f"l{i}.shift"])
        mixer = {"channel_delta": channel_delta_mixer, "parallel": parallel_mixer}[spec["type"]]
        x = x + mixer(h, sub(f"l{i}.mix."), spec["mixer"], eps) * W[f"l{i}.ls1"]
        m = spec["mlp"]
        if m is not None:
            h, w = norm(f"l{i}.norm2", x), sub(f"l{i}.mlp.")
            x = x + (gelu_feed_forward(h, w) if m["kind"] == "dense" else mixture(h, w, m)) * W[f"l{i}.ls2"]
        if trace is not None:
            trace.append(x.clone())
    return norm("final.norm", x) @ W["head"].t()

"""Plain statements of the hybrid decoder's mechanisms, one function each, in the slowest readable form.

Everything here works on one sequence, token by token, in float64 by default, and shares no code with the package:
the tests compare the framework (prompts, portions, batches, decoding) with ``run_model``.
"""
from __future__ import annotations

import math

import torch


def dyn_tanh(x, alpha, weight, bias):
    """Norm without statistics: tanh(alpha x) scaled and shifted per channel."""
    return torch.tanh(alpha * x) * weight + bias


def silu(x):
    return x / (1.0 + torch.exp(-x))


def clamped_glu(gate, up, limit):
    """gate is cut from above, up on both sides; (up + 1) times gate's soft step with slope 1.702."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)


def linear(x, w, b=None):
    y = x @ w.t()
    return y if b is None else y + b


def embedding(tokens, table, scale):
    return table[torch.as_tensor(tokens, dtype=torch.long)] * scale


def causal_conv(x, taps):
    """x [T, C], taps [C, K]; the last column weighs the current token, rows before the start are zero."""
    T, _ = x.shape
    K = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for k in range(K):
            s = t - (K - 1) + k
            if s >= 0:
                y[t] += taps[:, k] * x[s]
    return y


def unit_vector(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def softplus(x):
    return torch.where(x > 0, x, torch.zeros_like(x)) + torch.log1p(torch.exp(-x.abs()))


def delta_recurrence(q, k, v, decay, beta, state=None):
    """q, k [T, H, D], v [T, H, E], decay, beta [T, H]; state [H, D, E]. Returns (o [T, H, E], state)."""
    T, H, D = q.shape
    E = v.shape[-1]
    S = torch.zeros(H, D, E, dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, E, dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = S[h] * decay[t, h]
            seen = S[h].t() @ k[t, h]
            u = beta[t, h] * (v[t, h] - seen)
            S[h] = S[h] + torch.outer(k[t, h], u)
            out[t, h] = S[h].t() @ q[t, h]
    return out, S


def gated_head_norm(o, gate, weight, eps):
    """o, gate [T, H, E]: every head over its root mean square, times a shared weight, times silu(gate)."""
    r = torch.sqrt((o * o).mean(-1, keepdim=True) + eps)
    return o / r * weight * silu(gate)


def delta_mixer(h, w, m, eps):
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(linear(h, w["q"]), w["q.conv"])).view(T, G, D)
    k = silu(causal_conv(linear(h, w["k"]), w["k.conv"])).view(T, G, D)
    v = silu(causal_conv(linear(h, w["v"]), w["v.conv"])).view(T, H, E)
    q = unit_vector(q) * D ** -0.5
    k = unit_vector(k)
    q = q.repeat_interleave(H // G, dim=1)
    k = k.repeat_interleave(H // G, dim=1)
    beta = 1.0 / (1.0 + torch.exp(-linear(h, w["b"])))
    decay = torch.exp(-torch.exp(w["A_log"]) * softplus(linear(h, w["a"]) + w["dt_bias"]))
    o, _ = delta_recurrence(q, k, v, decay, beta)
    o = gated_head_norm(o, linear(h, w["g"]).view(T, H, E), w["norm"], eps)
    return linear(o.reshape(T, H * E), w["o"])


def chunked_attention(q, k, v, scale, size):
    """q [T, H, D], k [T, G, D], v [T, G, E]; token i sees the tokens j <= i of its own run of ``size`` positions."""
    T, H, _ = q.shape
    G, E = k.shape[1], v.shape[2]
    out = torch.zeros(T, H, E, dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t()) * scale
        i = torch.arange(T)[:, None]
        j = torch.arange(T)[None, :]
        seen = (j <= i) & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))
        s = s.masked_fill(~seen, -math.inf)
        p = torch.exp(s - s.max(dim=1, keepdim=True).values)
        out[:, h] = (p / p.sum(1, keepdim=True)) @ v[:, g]
    return out


def attention_mixer(h, w, m):
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w["q"], w["q.b"]).view(T, H, D)
    k = linear(h, w["k"], w["k.b"]).view(T, G, D)
    v = linear(h, w["v"], w["v.b"]).view(T, G, E)
    o = chunked_attention(q, k, v, m["scale"], m["mask"]["size"])
    return linear(o.reshape(T, H * E), w["o"])


def feed_forward(h, w, limit):
    y = clamped_glu(linear(h, w["gate"], w["gate.b"]), linear(h, w["up"], w["up.b"]), limit)
    return linear(y, w["down"], w["down.b"])


def run_model(config, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one whole sequence. ``trace`` (a list) receives the residual after every layer run."""
    W = {n: t.to(dtype) for n, t in weights.items()}

    def sub(prefix):
        return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}

    def norm(name, x):
        return dyn_tanh(x, W[name + ".alpha"], W[name], W[name + ".b"])

    eps = config["norm"]["eps"]
    e = embedding(tokens, W["embed"], config["embedding"]["scale"])
    x = e.clone()

    def layer(i, x):
        spec = config["layers"][i]
        h = norm(f"l{i}.norm1", x)
        w = sub(f"l{i}.mix.")
        y = delta_mixer(h, w, spec["mixer"], eps) if spec["type"] == "delta" else attention_mixer(h, w, spec["mixer"])
        x = x + norm(f"l{i}.norm1b", y)
        if spec["mlp"] is not None:
            y = feed_forward(norm(f"l{i}.norm2", x), sub(f"l{i}.mlp."), spec["mlp"]["limit"])
            x = x + norm(f"l{i}.norm2b", y)
        if trace is not None:
            trace.append(x.clone())
        return x

    loop = config.get("loop")
    n = len(config["layers"])
    start, stop, times = (loop["start"], loop["stop"], loop["times"]) if loop else (n, n, 0)
    for i in range(start):
        x = layer(i, x)
    for t in range(times):
        if t > 0:
            x = x + e
        x = x + W["loop.step"][t]
        for i in range(start, stop):
            x = layer(i, x)
    for i in range(stop, n):
        x = layer(i, x)
    return norm("final.norm", x) @ W["embed"].t()

"""Plain statements of Vobotar's mechanisms, one function each, in the slowest readable form: one sequence at a time, in
float64 by default, sharing no code with the package. Mechanisms that other designs also have come from
``hybrid_oracle`` and ``polosun_oracle``."""
from __future__ import annotations

import math

import torch

from hybrid_oracle import causal_conv, linear, silu, softplus
from polosun_oracle import feed_forward, gelu_tanh, over_rms, rotate, sigmoid


def one_plus_rms_norm(x, w, eps):
    return over_rms(x, eps) * (1.0 + w)


def rotate_pairs(x, positions, rot):
    """x [T, ..., D]: neighbours (2i, 2i + 1) of the first ``dims`` coordinates turn together; the rest passes."""
    n, base = rot["dims"], rot["base"]
    y = x.clone()
    for t, p in enumerate(positions):
        for i in range(n // 2):
            a = p * base ** (-2.0 * i / n)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            y[t, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            y[t, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return y


# ------------------------------------------------------------------------------------------ attention
def distance_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def attend(q, k, v, scale, window=None, softcap=None, slopes=None, sink=None, one=False):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]. ``sink`` [H]: scores of a place without a key or value; ``one``: 1 more in
    the denominator."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    hidden = j > i
    if window is not None:
        hidden = hidden | (i - j >= window)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].t()) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if slopes is not None:
            s = s - slopes[h] * (i - j).to(s.dtype)
        s = s.masked_fill(hidden, -math.inf)
        top = s.max(dim=1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[h])
        if one:
            top = torch.clamp(top, min=0.0)
        p = torch.exp(s - top)
        den = p.sum(1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - top)
        if one:
            den = den + torch.exp(-top)
        out[:, h] = (p / den) @ v[:, h // per]
    return out


def biased_window_attention(h, w, m, eps):
    """Values are the keys before their norm; unit queries and keys; distances bias the scores; a sink per head; a gate per head."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = linear(h, w["q"], w["q.b"]).view(T, H, D)
    k = linear(h, w["k"], w["k.b"]).view(T, G, D)
    o = attend(over_rms(q, eps), over_rms(k, eps), k, m["scale"], window=m["mask"]["size"], slopes=distance_slopes(H), sink=w["sink"])
    o = o * sigmoid(linear(h, w["g"]))[:, :, None]
    return linear(o.reshape(T, -1), w["o"])


def rotary_window_attention(h, w, m, eps):
    """Query and key norm over the whole projection, half-split rotation, a gate per head."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = over_rms(linear(h, w["q"], w["q.b"]), eps) * w["q.norm"]
    k = over_rms(linear(h, w["k"], w["k.b"]), eps) * w["k.norm"]
    v = linear(h, w["v"], w["v.b"]).view(T, G, E)
    q, k = (rotate(t.view(T, -1, D), range(T), m["rot"]) for t in (q, k))
    o = attend(q, k, v, m["scale"], window=m["mask"]["size"])
    o = o * sigmoid(linear(h, w["g"]))[:, :, None]
    return linear(o.reshape(T, -1), w["o"])


def capped_attention(h, w, m, eps, first_values=None):
    """Norms per head, neighbours rotated, capped scores, one more in the denominator, a gate per element. Returns (result, values of
    this layer): ``first_values`` are mixed in where given."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = over_rms(linear(h, w["q"]).view(T, H, D), eps) * w["q.norm"]
    k = over_rms(linear(h, w["k"]).view(T, G, D), eps) * w["k.norm"]
    v = linear(h, w["v"]).view(T, G, E)
    if first_values is not None:
        v = (1.0 - w["vmix"]) * v + w["vmix"] * first_values
    q, k = (rotate_pairs(t, range(T), m["rot"]) for t in (q, k))
    o = attend(q, k, v, m["scale"], softcap=m["softcap"], one=True)
    return linear(o.reshape(T, -1) * sigmoid(linear(h, w["g"])), w["o"]), v


# ------------------------------------------------------------------------------------------ time mixing with channel decays
def shifted_mix(h, mu, last=None):
    before = torch.cat([torch.zeros_like(h[:1]) if last is None else last[None], h[:-1]])
    return h + (before - h) * mu


def bonus_recurrence(r, k, v, w, u, state=None):
    """r, k, w [T, H, D], v [T, H, E], u [H, D]; state [H, D, E]. Returns (o [T, H, E], state)."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=r.dtype)
    for t in range(T):
        new = k[t][:, :, None] * v[t][:, None, :]
        out[t] = ((S + u[:, :, None] * new) * r[t][:, :, None]).sum(1)
        S = w[t][:, :, None] * S + new
    return out, S


def time_mixer(h, w, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    mix = {s: shifted_mix(h, w["mu." + s]) for s in "rkvgw"}
    r, k, v = (linear(mix[s], w[s]).view(T, H, D) for s in "rkv")
    gate = silu(linear(mix["g"], w["g"]))
    decay = torch.exp(-torch.exp(linear(torch.tanh(linear(mix["w"], w["w1"])), w["w2"]) + w["w0"])).view(T, H, D)
    o, _ = bonus_recurrence(r, k, v, decay, w["u"])
    return linear(over_rms(o, eps).reshape(T, -1) * w["norm"] * gate, w["o"])


# ------------------------------------------------------------------------------------------ state-space duality
def ssd_recurrence(x, B, C, dt, a_log, D, state=None):
    """x [T, H, E], B, C [T, H, N], dt [T, H] (positive), a_log, D [H]; state [H, N, E]. Returns (y [T, H, E], state)."""
    T, H, E = x.shape
    S = torch.zeros(H, B.shape[-1], E, dtype=x.dtype) if state is None else state.clone()
    out = torch.zeros_like(x)
    for t in range(T):
        decay = torch.exp(-torch.exp(a_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = (S * C[t][:, :, None]).sum(1) + D[:, None] * x[t]
    return out, S


def gated_group_norm(y, z, weight, groups, eps):
    g = (y * silu(z)).view(y.shape[0], groups, -1)
    return over_rms(g, eps).reshape(y.shape) * weight


def ssd_mixer(h, w, m, eps):
    T, H, E, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * E
    p = linear(h, w["in"])
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"]) + w["conv.b"])
    x = xbc[:, :inner].view(T, H, E)
    B, C = (xbc[:, inner + s * G * N:inner + (s + 1) * G * N].view(T, G, N).repeat_interleave(H // G, dim=1) for s in (0, 1))
    y, _ = ssd_recurrence(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return linear(gated_group_norm(y.reshape(T, inner), z, w["norm"], m["norm_groups"], eps), w["o"])


# ------------------------------------------------------------------------------------------ the model
def token_side_input(x, e, w, eps):
    """e [T, dim]: what the side table holds for this layer and every token."""
    y = linear(gelu_tanh(linear(x, w["gate"])) * e, w["proj"])
    return x + over_rms(y, eps) * w["norm"]


def run_model(config, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one whole sequence. ``trace`` (a list) receives what every layer hands on."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps, side = config["norm"]["eps"], config["token_side"]["dim"]
    toks = torch.as_tensor(tokens, dtype=torch.long)

    def sub(prefix):
        return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}

    x = W["embed"][toks] * config["embedding"]["scale"]
    first = None
    for i, spec in enumerate(config["layers"]):
        w, m = sub(f"l{i}.mix."), spec["mixer"]
        if spec["type"] == "attention":
            y, v = capped_attention(x, w, m, eps, first if m["v_mix"] else None)
            if m["v_mix"] and first is None:
                first = v
        else:
            left, right = sub(f"l{i}.mix.left."), sub(f"l{i}.mix.right.")
            if spec["type"] == "parallel":
                a, b = biased_window_attention(x, left, m["left"], eps), time_mixer(x, right, m["right"], eps)
            else:
                a, b = rotary_window_attention(x, left, m["left"], eps), ssd_mixer(x, right, m["right"], eps)
            y = m["left_scale"] * a + m["right_scale"] * b
        x = x + one_plus_rms_norm(y, W[f"l{i}.norm1"], eps)
        if spec["mlp"] is not None:
            x = x + one_plus_rms_norm(feed_forward(x, sub(f"l{i}.mlp.")), W[f"l{i}.norm2"], eps)
        x = token_side_input(x, W["side.embed"][toks][:, i * side:(i + 1) * side], sub(f"l{i}.side."), eps)
        if trace is not None:
            trace.append(x.clone())
    return one_plus_rms_norm(x, W["final.norm"], eps) @ W["embed"].t()

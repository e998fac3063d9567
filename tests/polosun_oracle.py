"""Plain statements of Polosun's mechanisms, one function each, in the slowest readable form: one sequence at a time, in
float64 by default, sharing no code with the package. Mechanisms that other designs also have come from
``hybrid_oracle``."""
from __future__ import annotations

import math

import torch

from hybrid_oracle import causal_conv, linear, silu, softplus


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def over_rms(x, eps):
    """Every row over its root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_rms_norm(x, gain, eps):
    return over_rms(x, eps) * gain


# ------------------------------------------------------------------------------------------ positions
def rotary_frequencies(rot):
    """([dims / 2] angle per position, factor on cos and sin)."""
    n, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if s is None:
        return freq, 1.0

    def where(turns):       # index of the pair that makes this many turns over the original length
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(where(s["fast"])), 0)
    hi = min(math.ceil(where(s["slow"])), n - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, ..., D]: coordinate i of the first ``dims`` turns with coordinate i + dims / 2; the rest passes."""
    freq, mult = rotary_frequencies(rot)
    half = rot["dims"] // 2
    y = x.clone()
    for t, p in enumerate(positions):
        for i in range(half):
            c, s = mult * math.cos(p * freq[i]), mult * math.sin(p * freq[i])
            u, v = x[t, ..., i], x[t, ..., i + half]
            y[t, ..., i] = u * c - v * s
            y[t, ..., i + half] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------ latent attention
def latent_attention(q, q_rot, c, k_rot, w_uk, w_uv, scale):
    """q [T, H, D], q_rot [T, H, R], c [T, C], k_rot [T, R]; w_uk [H, D, C], w_uv [H, E, C]. Keys and values of every head are
    written out; token i sees the tokens j <= i."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, w_uv.shape[1], dtype=q.dtype)
    hidden = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    for h in range(H):
        k = c @ w_uk[h].t()
        v = c @ w_uv[h].t()
        s = (q[:, h] @ k.t() + q_rot[:, h] @ k_rot.t()) * scale
        s = s.masked_fill(hidden, -math.inf)
        p = torch.exp(s - s.max(dim=1, keepdim=True).values)
        out[:, h] = (p / p.sum(1, keepdim=True)) @ v
    return out


def latent_mixer(h, w, m, eps):
    T = h.shape[0]
    H, D, R, E, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = {**m["rot"], "dims": R}
    q = linear(h, w["q"]).view(T, H, D + R)
    down = linear(h, w["dkv"])
    c = over_rms(down[:, :C], eps) * w["dkv.norm"]
    k_rot = rotate(down[:, C:], range(T), rot)
    o = latent_attention(q[..., :D], rotate(q[..., D:], range(T), rot), c, k_rot, w["uk"].view(H, D, C), w["uv"].view(H, E, C),
                         m["scale"])
    return linear(o.reshape(T, H * E) * sigmoid(linear(h, w["g"])), w["o"])


# ------------------------------------------------------------------------------------------ retention
def retention(q, k, v, decay, state=None):
    """q, k [T, H, D] (rotated and scaled), v [T, H, E], decay [H]; state [H, D, E]. Returns (o [T, H, E], state)."""
    T, H, D = q.shape
    E = v.shape[-1]
    S = torch.zeros(H, D, E, dtype=q.dtype) if state is None else state.clone()
    g = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    out = torch.zeros(T, H, E, dtype=q.dtype)
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def retention_mixer(h, w, m, eps):
    T = h.shape[0]
    H, D, E = m["heads"], m["dim"], m["vdim"]
    q = rotate(linear(h, w["q"]).view(T, H, D), range(T), m["rot"])
    k = rotate(linear(h, w["k"]).view(T, H, D), range(T), m["rot"]) * D ** -0.5
    o, _ = retention(q, k, linear(h, w["v"]).view(T, H, E), m["decay"])
    return linear(over_rms(o, eps).reshape(T, H * E) * silu(linear(h, w["g"])), w["o"])


# ------------------------------------------------------------------------------------------ real-gated linear recurrence
def block_linear(u, w, b):
    """u [T, N * K] in N parts, each through its own square matrix w [N, out, in] and bias b [N, out]."""
    T = u.shape[0]
    N, K, _ = w.shape
    parts = [u[:, n * K:(n + 1) * K] @ w[n].t() + b[n] for n in range(N)]
    return torch.cat(parts, dim=1)


def gated_recurrence(u, r, i, lam, state=None):
    """u, r, i [T, W] (gates already between 0 and 1), lam [W]; state [W]. Returns (S of every token, last S)."""
    S = torch.zeros_like(u[0]) if state is None else state.clone()
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        a = torch.exp(log_a)
        S = a * S + torch.sqrt(1.0 - a * a) * i[t] * u[t]
        out[t] = S
    return out, S


def rglru_mixer(h, w):
    y = gelu_tanh(linear(h, w["y"], w["y.b"]))
    u = causal_conv(linear(h, w["x"], w["x.b"]), w["conv"]) + w["conv.b"]
    r = sigmoid(block_linear(u, w["ra"], w["ra.b"]))
    i = sigmoid(block_linear(u, w["ri"], w["ri.b"]))
    s, _ = gated_recurrence(u, r, i, w["lam"])
    return linear(s * y, w["o"])


# ------------------------------------------------------------------------------------------ the model
def feed_forward(h, w):
    return linear(silu(linear(h, w["gate"])) * linear(h, w["up"]), w["down"])


def depth_average(history, weights):
    x = torch.zeros_like(history[0])
    for j, past in enumerate(history):
        x = x + weights[j] * past
    return x


def run_model(config, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one whole sequence. ``trace`` (a list) receives what every layer hands on."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]

    def sub(prefix):
        return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}

    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    history = [x]
    for i, spec in enumerate(config["layers"]):
        w = sub(f"l{i}.mix.")
        h = scalar_rms_norm(x, W[f"l{i}.norm1"], eps)
        if spec["type"] == "latent_attention":
            y = latent_mixer(h, w, spec["mixer"], eps)
        elif spec["type"] == "retention":
            y = retention_mixer(h, w, spec["mixer"], eps)
        else:
            y = rglru_mixer(h, w)
        if spec["mlp"] is not None:
            y = y + feed_forward(scalar_rms_norm(x, W[f"l{i}.norm2"], eps), sub(f"l{i}.mlp."))
        history.append(x + m * y)
        x = depth_average(history, W[f"l{i}.dwa"])
        if trace is not None:
            trace.append(x.clone())
    return scalar_rms_norm(x, W["final.norm"], eps) @ W["head"].t()

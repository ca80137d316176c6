"""A plain, slow statement of the Rasezen decoder: whole sequences, no cache, float64, one function per mechanism.

It shares no code with the package: the configuration is the config.json dictionary and the weights a dictionary of
checkpoint names to tensors.  The state mixer walks its tokens one by one and keeps the state as an explicit matrix, every
query has its own softmax row over a boolean mask, and every expert is evaluated for the tokens that chose it, one at a time.
"""

from __future__ import annotations

import math

import torch

F = torch.float64
ROUND = None  # a dtype, or a function of a tensor: activations pass through it wherever a 16-bit pipeline would store them


def r(t):
    """What a reduced-precision pipeline keeps of an activation; the identity unless `ROUND` is set."""
    if ROUND is None:
        return t
    return ROUND(t) if callable(ROUND) else t.to(ROUND).to(F)


def rms_norm(x, eps, g):
    """x over the root of its mean square (eps inside the root), times g: one number or one per feature."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * g


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def xielu(z, p, q):
    """A quadratic branch for z > 0 and an exponential one for z <= 0, both with slope 1/2 at zero."""
    return torch.where(z > 0, softplus(p) * z * z + 0.5 * z,
                       (0.5 + softplus(q)) * (torch.exp(torch.clamp(z, max=0.0)) - 1.0 - z) + 0.5 * z)


def rotate_half(x, positions, dims, base):
    """x [T, heads, dim]: features i and i + dims/2 turn by position * base^(-2i/dims), i < dims/2; the rest pass."""
    if dims == 0:
        return x
    n = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(n)], dtype=F)
    ang = (positions.to(F)[:, None] * f[None, :])[:, None, :]
    u, v = x[..., :n], x[..., n:dims]
    out = x.clone()
    out[..., :n] = u * torch.cos(ang) - v * torch.sin(ang)
    out[..., n:dims] = v * torch.cos(ang) + u * torch.sin(ang)
    return out


def window_mask(T, size):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def attend(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        out[:, h] = torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1) @ v[:, g]
    return out.reshape(T, -1)


def mixer_attention(h, m, W, pre, eps, positions):
    """Biases on q, k and v, one RMS norm over the whole q and the whole k projection, rotation in halves, values divided by
    their root mean square per head, a sliding window."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = r(h @ W[pre + "q"].T) + W[pre + "q.b"]
    k = r(h @ W[pre + "k"].T) + W[pre + "k.b"]
    v = r(h @ W[pre + "v"].T) + W[pre + "v.b"]
    q = rms_norm(q, eps, W[pre + "q.norm"]).view(T, H, d)
    k = rms_norm(k, eps, W[pre + "k.norm"]).view(T, G, d)
    rot = m["rot"]
    q = r(rotate_half(q, positions, int(rot["dims"]), float(rot["base"])))
    k = r(rotate_half(k, positions, int(rot["dims"]), float(rot["base"])))
    v = r(rms_norm(v.view(T, G, dv), eps, 1.0))
    o = r(attend(q, k, v, float(m["scale"]), window_mask(T, int(m["mask"]["size"]))))
    return r(o @ W[pre + "o"].T)


def causal_convolution(u, w, b):
    """u [T, C], w [C, taps], b [C]: y_t = b + sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = b[None, :].repeat(T, 1)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * u[s]
    return y


def state_space_walk(x, B, C, dt, a_log, D):
    """x [T, H, V], B and C [T, G, N], dt [T, H] (after the softplus).  Per head, from S = 0:
    S = exp(-exp(a_log) dt_t) S + dt_t B_t x_t^T,  y_t = S^T C_t + D x_t.  Returns y [T, H, V]."""
    T, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    y = torch.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(N, V, dtype=x.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + D[h] * x[t, h]
    return y


def gated_norm(y, z, eps, g, parts):
    """y silu(z), then each of `parts` equal runs of features over its own root mean square, times g."""
    u = y * silu(z)
    T, inner = u.shape
    u = u.view(T, parts, inner // parts)
    return (u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)).reshape(T, inner) * g


def mixer_mamba2(h, m, W, pre, eps, positions):
    """One projection [z | x | B | C | dt]; x, B and C through a short convolution and silu; the state's walk; the gate, then
    the norm in equal parts; the output projection."""
    T = h.shape[0]
    H, V, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * V
    p = r(h @ W[pre + "in"].T)
    z, xbc, dt = p[:, :inner], p[:, inner: 2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = r(silu(causal_convolution(xbc, W[pre + "conv"], W[pre + "conv.b"])))
    x, B, C = xbc[:, :inner], xbc[:, inner: inner + G * N], xbc[:, inner + G * N:]
    dt = softplus(dt + W[pre + "dt_bias"])
    y = state_space_walk(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, W[pre + "A_log"], W[pre + "D"])
    u = r(gated_norm(y.reshape(T, inner), z, eps, W[pre + "norm"], int(m["norm_groups"])))
    return r(u @ W[pre + "o"].T)


MIXERS = {"attention": mixer_attention, "mamba2": mixer_mamba2}


def dense(h, W, pre):
    p, q = W[pre + "act"][0], W[pre + "act"][1]
    return r(r(xielu(r(h @ W[pre + "up"].T), p, q)) @ W[pre + "down"].T)


def expert(h, W, pre):
    return r(r(silu(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T)


def route(h, router, W, pre):
    """(chosen [T, top], weights [T, top]): softmax scores over every expert, the ones that return their input included; the
    choice by score plus correction; the weights are the bare scores times the router's scale."""
    s = torch.softmax(h @ W[pre + "router"].T, dim=-1)
    chosen = torch.argsort(s + W[pre + "correction"], dim=-1, descending=True, stable=True)[:, : int(router["top"])]
    return chosen, s.gather(1, chosen) * float(router["scale"])


def mixture(h, mlp, W, pre):
    router = mlp["router"]
    chosen, weights = route(h, router, W, pre)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            y[t] = y[t] + w * (expert(h[t: t + 1], W, f"{pre}e{e}.")[0] if e < int(router["experts"]) else h[t])
    y = r(y)
    if mlp.get("shared") is not None:
        y = y + expert(h, W, pre + "shared.")
    return y


def feed_forward(h, mlp, W, pre):
    return dense(h, W, pre) if mlp["kind"] == "dense" else mixture(h, mlp, W, pre)


def forward(cfg: dict, weights: dict, tokens, rounded=None, layers_out: list | None = None):
    """tokens: a list of ids of one sequence -> float64 logits [T, vocab].  `layers_out` receives the stream after each layer."""
    global ROUND
    ROUND = rounded
    try:
        W = {k: torch.as_tensor(v).to(F) for k, v in weights.items()}
        eps = float(cfg["norm"]["eps"])
        ids = torch.as_tensor(tokens, dtype=torch.long)
        positions = torch.arange(len(ids))
        x = W["embed"][ids]
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            h = r(rms_norm(x, eps, W[p + "norm1"]))
            y = MIXERS[layer["type"]](h, layer["mixer"], W, p + "mix.", eps, positions)
            if layer.get("mlp") is not None:
                y = y + feed_forward(h, layer["mlp"], W, p + "mlp.")
            x = x + y
            if layers_out is not None:
                layers_out.append(x.clone())
        return r(rms_norm(x, eps, W["final.norm"])) @ W["head"].T
    finally:
        ROUND = None

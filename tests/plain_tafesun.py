"""A plain, slow statement of the Tafesun decoder: whole sequences, no cache, float64, one function per mechanism.

It shares no code with the package: the configuration is the config.json dictionary and the weights a dictionary of
checkpoint names to tensors.  The state space walks its tokens one by one and keeps the state as an explicit matrix per head, every
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


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def dynamic_tanh(x, W, name):
    """tanh(alpha x), one number alpha, then a gain and a bias per feature; no statistics."""
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def frequencies(rot):
    """One angle per position for each of the dims / 2 pairs; `scaling.factor` slows all of them alike."""
    n, dims = int(rot["dims"]) // 2, int(rot["dims"])
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    return torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) / factor for i in range(n)], dtype=F)


def rotate_half(x, positions, rot):
    """x [T, heads, dim]: features i and i + dims/2 turn together, i < dims/2; the rest pass."""
    dims = int(rot["dims"])
    if dims == 0:
        return x
    n = dims // 2
    ang = (positions.to(F)[:, None] * frequencies(rot)[None, :])[:, None, :]
    u, v = x[..., :n], x[..., n:dims]
    out = x.clone()
    out[..., :n] = u * torch.cos(ang) - v * torch.sin(ang)
    out[..., n:dims] = v * torch.cos(ang) + u * torch.sin(ang)
    return out


def attend(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv]; causal; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        out[:, h] = torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1) @ v[:, g]
    return out.reshape(T, -1)


def attention_half(h, m, W, pre, positions):
    """Biases on q, k and v; rotation in halves; every earlier key; each output feature times the sigmoid of its own gate."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (r(h @ W[pre + "q"].T) + W[pre + "q.b"]).view(T, H, d)
    k = (r(h @ W[pre + "k"].T) + W[pre + "k.b"]).view(T, G, d)
    v = r(r(h @ W[pre + "v"].T) + W[pre + "v.b"]).view(T, G, dv)
    q, k = r(rotate_half(q, positions, m["rot"])), r(rotate_half(k, positions, m["rot"]))
    gate = sigmoid(r(h @ W[pre + "g"].T))
    return attend(q, k, v, float(m["scale"])) * gate


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
    of = torch.tensor([h // (H // G) for h in range(H)])
    y = torch.zeros_like(x)
    S = torch.zeros(H, N, V, dtype=x.dtype)
    for t in range(T):
        write = B[t, of][:, :, None] * x[t][:, None, :]
        S = torch.exp(-torch.exp(a_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * write
        y[t] = (S * C[t, of][:, :, None]).sum(1) + D[:, None] * x[t]
    return y


def gated_norm(y, z, eps, g, parts):
    """y silu(z), then each of `parts` equal runs of features over its own root mean square, times g."""
    u = y * silu(z)
    T, inner = u.shape
    u = u.view(T, parts, inner // parts)
    return (u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)).reshape(T, inner) * g


def state_space_half(h, m, W, pre, eps):
    """One projection [z | x | B | C | dt]; x, B and C through a short convolution and silu; the state's walk; the gate, then
    the norm in equal parts."""
    T = h.shape[0]
    H, V, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * V
    p = r(h @ W[pre + "in"].T)
    z, xbc, dt = p[:, :inner], p[:, inner: 2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = r(silu(causal_convolution(xbc, W[pre + "conv"], W[pre + "conv.b"])))
    x, B, C = xbc[:, :inner], xbc[:, inner: inner + G * N], xbc[:, inner + G * N:]
    dt = softplus(dt + W[pre + "dt_bias"])
    y = state_space_walk(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, W[pre + "A_log"], W[pre + "D"])
    return gated_norm(y.reshape(T, inner), z, eps, W[pre + "norm"], int(m["norm_groups"]))


def mixer_parallel(h, m, W, pre, eps, positions):
    """Attention and the state space on the same input, each with its output projection, added with constant weights."""
    a = r(attention_half(h, m["left"], W, pre + "left.", positions)) @ W[pre + "left.o"].T
    b = r(state_space_half(h, m["right"], W, pre + "right.", eps)) @ W[pre + "right.o"].T
    return r(float(m["left_scale"]) * a + float(m["right_scale"]) * b)


def expert(h, W, pre, limit):
    """g from above and u from both sides held within `limit`; g sigmoid(1.702 g) (u + 1), then the way down."""
    g = torch.clamp(h @ W[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ W[pre + "up"].T, min=-limit, max=limit)
    return r(g * sigmoid(1.702 * g) * (u + 1.0)) @ W[pre + "down"].T


def route(h, router, W, pre):
    """(chosen [T, top], weights [T, top]): the largest biased logits, their softmax among themselves."""
    z = h @ W[pre + "router"].T + W[pre + "router.b"]
    chosen = torch.argsort(z, dim=-1, descending=True, stable=True)[:, : int(router["top"])]
    return chosen, torch.softmax(z.gather(1, chosen), dim=-1)


def mixture(h, mlp, W, pre):
    chosen, weights = route(h, mlp["router"], W, pre)
    limit = float(mlp["expert"]["limit"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            y[t] = y[t] + w * r(expert(h[t: t + 1], W, f"{pre}e{e}.", limit))[0]
    if mlp.get("shared") is not None:
        y = y + r(expert(h, W, pre + "shared.", float(mlp["shared"]["limit"])))
    return y


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = int(cfg["layers"][i]["weights_of"])
    return i


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
            p = f"l{owner(cfg, i)}."
            y = mixer_parallel(r(dynamic_tanh(x, W, p + "norm1")), layer["mixer"], W, p + "mix.", eps, positions)
            x = x + dynamic_tanh(y, W, p + "norm1b")
            if layer.get("mlp") is not None:
                y = mixture(r(dynamic_tanh(x, W, p + "norm2")), layer["mlp"], W, p + "mlp.")
                x = x + dynamic_tanh(y, W, p + "norm2b")
            if layers_out is not None:
                layers_out.append(x.clone())
        return (r(dynamic_tanh(x, W, "final.norm")) @ W["embed"].T) * float(cfg["logit_scale"])
    finally:
        ROUND = None

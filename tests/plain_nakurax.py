"""A plain, slow statement of the Nakurax design in 64-bit torch on the CPU: one function per mechanism, whole
sequences only, no cache.  The tests compare the library with it; it shares no code with the library.

Notation: h [T, W] is a sublayer's input (the weighted sum of the streams, normed), ``w`` a dict from tensor name (as the
model file spells it) to a 64-bit tensor, ``cfg`` the config.json dict, ``m`` a mixer's entry of it.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
    """One per pair of dims: base^(-2i/dims); with ``scaling`` those whose wavelength passes original/low are divided by
    the factor, those below original/high stay, those between are blended by how often they turn over ``original``."""
    n = int(rot["dims"])
    out = []
    for i in range(n // 2):
        f = float(rot["base"]) ** (-2.0 * i / n)
        sc = rot.get("scaling")
        if sc is not None:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif not wave < sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x, rot, first_position=0):
    """x [T, heads, dim]: dims 2i and 2i + 1 of every head, i below rot.dims / 2, turned by position * frequency i."""
    n = int(rot["dims"]) if rot else 0
    if n == 0:
        return x
    T = x.shape[0]
    angle = torch.arange(first_position, first_position + T, dtype=F64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    out = x.clone()
    a, b = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = a * c - b * s
    out[..., 1:n:2] = b * c + a * s
    return out


def softmax_rows(s):
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_attention(h, w, pre, m, eps):
    """Keys and values of every head are read out of a normed latent per position; all earlier positions are seen."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, D)
    c = rms(h @ w[pre + "dkv"].T, w[pre + "dkv.norm"], eps)
    k = (c @ w[pre + "uk"].T).view(T, H, D)
    v = (c @ w[pre + "uv"].T).view(T, H, V)
    seen = torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for head in range(H):
        s = (q[:, head] @ k[:, head].T * m["scale"]).masked_fill(~seen, -math.inf)
        out[:, head] = softmax_rows(s) @ v[:, head]
    return out.reshape(T, H * V) @ w[pre + "o"].T


def chunked_attention(h, w, pre, m):
    """Grouped softmax attention inside chunks of mask.size positions, counted from the sequence's start."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[pre + "q"].T).view(T, H, D), m.get("rot"))
    k = rotate((h @ w[pre + "k"].T).view(T, G, D), m.get("rot"))
    v = (h @ w[pre + "v"].T).view(T, G, V)
    pos = torch.arange(T)
    chunk = pos // int(m["mask"]["size"])
    seen = (pos[:, None] >= pos[None, :]) & (chunk[:, None] == chunk[None, :])
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T * m["scale"]).masked_fill(~seen, -math.inf)
        out[:, head] = softmax_rows(s) @ v[:, g]
    return out.reshape(T, H * V) @ w[pre + "o"].T


def causal_conv(x, taps_w, bias):
    """x [T, C]; taps_w [C, taps], the last column weighs the current token; zeros before the start."""
    T, C = x.shape
    taps = taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x], 0)
    y = bias.expand(T, C).clone()
    for j in range(taps):
        y = y + padded[j:j + T] * taps_w[:, j]
    return y


def block_gate(u, matrices, biases):
    """sigmoid of a product per equal part of the channels: matrices [blocks, size, size], biases [blocks, size]."""
    T, C = u.shape
    blocks, size = biases.shape
    parts = u.view(T, blocks, size)
    return torch.sigmoid(torch.stack([parts[:, b] @ matrices[b].T + biases[b] for b in range(blocks)], 1)).reshape(T, C)


def gated_recurrence(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t from zero, log a_t = -8 r_t softplus(lam)."""
    log_a = -8.0 * r * torch.log1p(torch.exp(lam))
    S = torch.zeros(u.shape[1], dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        a = torch.exp(log_a[t])
        S = a * S + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * i[t] * u[t]
        out[t] = S
    return out


def recurrent_block(h, w, pre, m):
    y = gelu_tanh(h @ w[pre + "y"].T + w[pre + "y.b"])
    u = causal_conv(h @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    r = block_gate(u, w[pre + "ra"], w[pre + "ra.b"])
    i = block_gate(u, w[pre + "ri"], w[pre + "ri.b"])
    return (gated_recurrence(u, r, i, w[pre + "lam"]) * y) @ w[pre + "o"].T


def parallel_mixer(h, w, pre, m, eps):
    return (m["left_scale"] * chunked_attention(h, w, pre + "left.", m["left"])
            + m["right_scale"] * recurrent_block(h, w, pre + "right.", m["right"]))


def dense_ff(h, w, pre):
    return torch.relu(h @ w[pre + "up"].T) ** 2 @ w[pre + "down"].T


MIXERS = {"latent_attention": latent_attention, "parallel": parallel_mixer}


def hyper_connected(X, w, pre, sublayer):
    """X [streams, T, W]: the sublayer reads sum_s in_s X_s; stream t then holds sum_s mix_st X_s plus out_t times what the
    sublayer returned."""
    u = sum(w[pre + "in"][s] * X[s] for s in range(X.shape[0]))
    y = sublayer(u)
    return torch.stack([sum(w[pre + "mix"][s, t] * X[s] for s in range(X.shape[0])) + w[pre + "out"][t] * y
                        for t in range(X.shape[0])])


def run_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n))


def forward(tokens, w, cfg, keep_layers=False):
    """Logits [T, vocab] of one whole sequence (and the sum of the streams after every layer run)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    X = torch.stack([x] * int(cfg["streams"]))
    layers = []
    for i in run_order(cfg):
        L, pre = cfg["layers"][i], f"l{i}."
        X = hyper_connected(X, w, pre + "hc1.", lambda u: MIXERS[L["type"]](rms(u, w[pre + "norm1"], eps), w,
                                                                            pre + "mix.", L["mixer"], eps))
        if L.get("mlp") is not None:
            X = hyper_connected(X, w, pre + "hc2.", lambda u: dense_ff(rms(u, w[pre + "norm2"], eps), w, pre + "mlp."))
        if keep_layers:
            layers.append(X.sum(0))
    logits = rms(X.sum(0), w["final.norm"], eps) @ w["head"].T
    return (logits, layers) if keep_layers else logits

"""A plain, slow statement of the Dibedra design in 64-bit torch on the CPU: one function per mechanism, whole
sequences only, no cache.  The tests compare the library with it; it shares no code with the library.

Notation: h [T, W] is the input both sublayers of a layer read, ``w`` a dict from tensor name (as the model file
spells it) to a 64-bit tensor, ``cfg`` the config.json dict, ``m`` a mixer's entry of it, ``pre`` the prefix of a
sublayer's tensor names.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def dynamic_tanh(x, w, name):
    """A squashing in place of a norm: no statistics, one learned slope for all coordinates."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def pair_frequencies(rot):
    """(turns per position of every pair of dims, factor on cosine and sine)."""
    n, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return plain, 1.0
    # slow pairs (few turns over the original length) are stretched by the factor, fast ones stay, a ramp between
    place = lambda turns: n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    first = max(math.floor(place(s["fast"])), 0)
    last = min(math.ceil(place(s["slow"])), n - 1)
    out = []
    for i, f in enumerate(plain):
        slow = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * slow + f * (1.0 - slow))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, rot):
    """x [T, heads, dim]: dims 2i and 2i + 1 of every head turned together, the dims behind rot.dims stay."""
    n = int(rot["dims"]) if rot else 0
    if n == 0:
        return x
    freq, gain = pair_frequencies(rot)
    angle = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(freq, dtype=F64)[None, :]
    c, s = gain * torch.cos(angle)[:, None, :], gain * torch.sin(angle)[:, None, :]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], -1).reshape(*x.shape[:-1], n)
    return torch.cat([turned, x[..., n:]], -1)


def queries(h, w, pre, m, eps):
    q = (h @ w[pre + "q"].T).view(h.shape[0], m["heads"], m["dim"])
    return rotate_pairs(unit_rms(q, eps) * w[pre + "q.norm"], m.get("rot"))


def keys_and_values(h, w, pre, m, eps):
    """One projection gives both: the values are its rows as they are, the keys its rows normed and turned."""
    raw = (h @ w[pre + "k"].T).view(h.shape[0], m["kv_heads"], m["dim"])
    return rotate_pairs(unit_rms(raw, eps) * w[pre + "k.norm"], m.get("rot")), raw


def visible(T, m):
    """[T, T]: which positions j (columns) position i (rows) sees."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = back >= 0
    return seen & (back < int(m["mask"]["size"])) if m.get("mask") else seen


def attention(h, w, pre, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = queries(h, w, pre, m, eps)
    k, v = keys_and_values(h, w, pre, m, eps)
    seen = visible(T, m)
    out = torch.zeros(T, H, m["vdim"], dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"]
        out[:, head] = torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, g]
    gate = torch.sigmoid(h @ w[pre + "g"].T)
    return (out.reshape(T, -1) * gate) @ w[pre + "o"].T


def dense_ff(h, w, pre):
    return gelu_tanh(h @ w[pre + "up"].T) @ w[pre + "down"].T


def expert(h, w, pre, limit):
    g = torch.clamp(h @ w[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ w[pre + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def route(h, w, pre, r):
    """(chosen outputs of the router [T, top], their weights [T, top]).  Outputs from r.experts on are the identity."""
    n = int(r["experts"]) + int(r.get("identity") or 0)
    s = torch.softmax(h @ w[pre + "router"].T, -1)
    choice = s + w[pre + "correction"]
    groups = r.get("groups")
    if groups:
        per = n // int(groups["count"])
        by_group = choice.view(-1, int(groups["count"]), per)
        best = torch.topk(by_group.max(-1).values, int(groups["keep"]), dim=-1).indices
        stays = torch.zeros(by_group.shape[:2], dtype=torch.bool).scatter_(1, best, True)
        choice = by_group.masked_fill(~stays[..., None], -math.inf).reshape(-1, n)
    ids = torch.topk(choice, int(r["top"]), dim=-1).indices
    return ids, torch.gather(s, 1, ids)


def moe_ff(h, w, pre, mlp):
    r = mlp["router"]
    ids, weights = route(h, w, pre, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), weights[t]):
            y = h[t] if e >= r["experts"] else expert(h[t:t + 1], w, f"{pre}e{e}.", float(mlp["expert"]["limit"]))[0]
            out[t] += a * y
    return out


def forward(cfg, w, tokens, layer_outputs=None):
    """Logits [T, vocab] of one sequence; ``layer_outputs``: a list that receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)].to(F64)
    for i, L in enumerate(cfg["layers"]):
        if L["type"] != "attention":
            raise ValueError(f"unknown layer type {L['type']!r}")
        own = i
        while cfg["layers"][own].get("weights_of") is not None:
            own = cfg["layers"][own]["weights_of"]
        p = f"l{own}."
        h = dynamic_tanh(x, w, p + "norm1")
        y = attention(h, w, p + "mix.", L["mixer"], eps)
        mlp = L.get("mlp")
        if mlp is not None:
            y = y + (dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp))
        x = x + y
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return (dynamic_tanh(x, w, "final.norm") @ w["head"].T) * float(cfg["logit_scale"])

"""Zuvasun in plain, slow torch (float64 on the CPU): the oracle of the Zuvasun tests.

One function per mechanism, written from the design's equations; it shares no code with the package.  A model is a
configuration dict (the keys of the architecture's config.json) and a dict of tensors by the names of a model folder.
Attention expands every key and value and looks at them query by query; nothing is cached, absorbed or packed.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# --------------------------------------------------------------------------------------------- small pieces
def rmsnorm(x, gain, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * gain


def softmax_row(s):
    e = torch.exp(s - s.max())
    return e / e.sum()


def turning_speeds(rot):
    """(angle per position of every pair, factor on cos and sin) of a rotation {base, dims, scaling (optional)}."""
    dims, base = rot["dims"], float(rot["base"])
    speeds = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return speeds, 1.0

    def place(turns):           # the (fractional) pair that makes `turns` whole turns within the original length
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(sc["fast"])), 0)
    hi = min(math.ceil(place(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(speeds):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def turn_pairs(x, pos, rot):
    """x [..., dims]: value 2i turned with value 2i + 1 by pos * speed_i, both times the rotation's factor."""
    speeds, factor = turning_speeds(rot)
    out = x.clone()
    for i, f in enumerate(speeds):
        c, s = factor * math.cos(pos * f), factor * math.sin(pos * f)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def query_temperature(m, pos):
    t = m.get("q_temp")
    return 1.0 if t is None else 1.0 + t["coef"] * math.log(math.floor((pos + 1) / t["every"]) + 1)


# --------------------------------------------------------------------------------------------- mixers
def attention(h, p, m, eps):
    """Grouped-query attention without positions whose values are the projected keys."""
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = h @ p["q"].T + p["q.b"]
    k = h @ p["k"].T + p["k.b"]
    v = k.view(T, G, D)
    q = rmsnorm(q, p["q.norm"], eps).view(T, H, D)
    k = rmsnorm(k, p["k.norm"], eps).view(T, G, D)
    out = torch.zeros(T, H, D, dtype=h.dtype)
    for i in range(T):
        temp = query_temperature(m, i)
        for hh in range(H):
            g = hh // (H // G)
            w = softmax_row(k[:i + 1, g] @ (q[i, hh] * temp) * m["scale"])
            out[i, hh] = w @ v[:i + 1, g]
    return out.reshape(T, H * D) @ p["o"].T


def latent_entries(h, p, m, eps):
    """What a layer keeps of every token: the normed latent [T, rank] and the turned key part shared by all heads."""
    z = h @ p["dkv"].T
    c = rmsnorm(z[:, :m["kv_rank"]], p["dkv.norm"], eps)
    r = z[:, m["kv_rank"]:]
    return c, torch.stack([turn_pairs(r[t], t, m["rot"]) for t in range(h.shape[0])])


def latent_attention(h, p, m, entries):
    """`entries`: this layer's own latents and key parts, or those of the layer it reads."""
    T = h.shape[0]
    H, D, R, E = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = entries
    q = (h @ p["q"].T).view(T, H, D + R)
    kn = (c @ p["uk"].T).view(T, H, D)
    v = (c @ p["uv"].T).view(T, H, E)
    size = m["mask"]["size"] if m.get("mask") else None
    out = torch.zeros(T, H, E, dtype=h.dtype)
    for i in range(T):
        first = 0 if size is None else max(0, i - size + 1)
        qr = turn_pairs(q[i, :, D:], i, m["rot"])
        for hh in range(H):
            s = (kn[first:i + 1, hh] @ q[i, hh, :D] + kr[first:i + 1] @ qr[hh]) * m["scale"]
            out[i, hh] = softmax_row(s) @ v[first:i + 1, hh]
    return out.reshape(T, H * E) @ p["o"].T


# --------------------------------------------------------------------------------------------- feed-forward
def choose(z, correction, top, scale):
    """One token's router logits [E]: the chosen experts and their weights."""
    s = softmax_row(z)
    best = torch.topk(s + correction, top).indices.tolist()
    total = sum(float(s[e]) for e in best) + 1e-20
    return best, [float(s[e]) / total * scale for e in best]


def routed_ff(h, p, f):
    out = torch.zeros(h.shape[0], p["e0.down"].shape[0], dtype=h.dtype)
    for t in range(h.shape[0]):
        best, weights = choose(p["router"] @ h[t], p["correction"], f["router"]["top"], f["router"]["scale"])
        for e, w in zip(best, weights):
            out[t] += w * (p[f"e{e}.down"] @ torch.relu(p[f"e{e}.up"] @ h[t]) ** 2)
    return out


# --------------------------------------------------------------------------------------------- the model
def sub(tensors, prefix):
    return {n[len(prefix):]: t for n, t in tensors.items() if n.startswith(prefix)}


def forward(cfg, tensors, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token (float64), and, asked for, the stream after every layer."""
    tensors = {n: t.to(F64) for n, t in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = tensors["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kept, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        t, m = sub(tensors, f"l{i}."), layer["mixer"]
        p = sub(t, "mix.")
        h = rmsnorm(x, t["norm1"], eps)
        if layer["type"] == "attention":
            y = attention(h, p, m, eps)
        else:
            src = m.get("kv_from")
            if src is None:
                kept[i] = latent_entries(h, p, m, eps)
            y = latent_attention(h, p, m, kept[i if src is None else src])
        y = t["ls1"] * y
        if layer.get("mlp") is not None:
            y = y + t["ls2"] * routed_ff(h, sub(t, "mlp."), layer["mlp"])
        x = x + y
        after.append(x)
    logits = rmsnorm(x, tensors["final.norm"], eps) @ tensors["head"].T
    return (logits, torch.stack(after)) if return_layers else logits

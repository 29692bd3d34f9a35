"""Kugisun in plain, slow torch (float64 on the CPU): the oracle of the Kugisun tests.

One function per mechanism, written from the design's equations; it shares no code with the package.  A model is a
configuration dict (the keys of the architecture's config.json) and a dict of tensors by the names of a model folder.
Attention looks at every key query by query, the delta rule walks a sequence token by token; nothing is cached or packed.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


# --------------------------------------------------------------------------------------------- small pieces
def rmsnorm(x, gain, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * gain


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


def turn_neighbours(x, pos, rot):
    """x [..., d]: in the first rot.dims values, value 2i turned with value 2i + 1 by pos * base^(-2i/dims)."""
    out = x.clone()
    for i in range(rot["dims"] // 2):
        a = pos * float(rot["base"]) ** (-2.0 * i / rot["dims"])
        c, s = math.cos(a), math.sin(a)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def short_conv(u, taps):
    """u [T, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j), zeros before the first token."""
    T, K = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(K):
            s = t - K + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


# --------------------------------------------------------------------------------------------- mixers
def attention_heads(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e]: causal softmax over every key at or before the query."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        for h in range(H):
            g = h // (H // G)
            s = (k[:i + 1, g] @ q[i, h]) * scale
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[:i + 1, g]
    return out


def attention(h, p, m, eps):
    """The left branch.  h [T, W]; p: the branch's tensors by their last name."""
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rmsnorm((h @ p["q"].T + p["q.b"]).view(T, H, D), p["q.norm"], eps)
    k = rmsnorm((h @ p["k"].T + p["k.b"]).view(T, G, D), p["k.norm"], eps)
    v = (h @ p["v"].T + p["v.b"]).view(T, G, E)
    if m.get("rot"):
        q = torch.stack([turn_neighbours(q[t], t, m["rot"]) for t in range(T)])
        k = torch.stack([turn_neighbours(k[t], t, m["rot"]) for t in range(T)])
    return attention_heads(q, k, v, m["scale"]).reshape(T, H * E) @ p["o"].T


def delta_memory(q, k, v, beta, g, S=None):
    """q, k [T, G, d] (unit vectors, q scaled), v [T, H, e], beta and g [T, H]; S [H, d, e] or None for zeros.  Every token:
    S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  Returns every o and the last S."""
    T, H, E = v.shape
    G, D = k.shape[1], k.shape[2]
    S = torch.zeros(H, D, E, dtype=v.dtype) if S is None else S.clone()
    out = torch.zeros(T, H, E, dtype=v.dtype)
    for t in range(T):
        for h in range(H):
            kv = h // (H // G)
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, kv])
            S[h] = S[h] + torch.outer(k[t, kv], u)
            out[t, h] = S[h].T @ q[t, kv]
    return out, S


def gated_delta(h, p, m, eps):
    """The right branch."""
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(silu(short_conv(h @ p["q"].T, p["q.conv"])).view(T, G, D)) * D ** -0.5
    k = unit(silu(short_conv(h @ p["k"].T, p["k.conv"])).view(T, G, D))
    v = silu(short_conv(h @ p["v"].T, p["v.conv"])).view(T, H, E)
    beta = 1.0 / (1.0 + torch.exp(-(h @ p["b"].T)))
    g = torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o = rmsnorm(delta_memory(q, k, v, beta, g)[0], p["norm"], eps)
    return (o.reshape(T, H * E) * silu(h @ p["g"].T)) @ p["o"].T


def parallel_mixer(h, p, m, eps):
    return m["left_scale"] * attention(h, sub(p, "left."), m["left"], eps) + m["right_scale"] * gated_delta(h, sub(p, "right."), m["right"], eps)


# --------------------------------------------------------------------------------------------- feed-forwards
def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose(z, correction, r):
    """One token's router logits [experts + identity]: the chosen outputs and their weights.  Groups of neighbours, best
    choice score first; only outputs of the groups kept can be chosen."""
    e = torch.exp(z - z.max())
    s = (e / e.sum()).tolist()
    c = [a + float(b) for a, b in zip(s, correction)]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    size = len(c) // groups["count"]
    best_of = sorted(range(groups["count"]), key=lambda g: -max(c[g * size:(g + 1) * size]))
    kept = set(best_of[:groups["keep"]])
    able = [i for i in range(len(c)) if i // size in kept]
    best = sorted(able, key=lambda i: -c[i])[:r["top"]]
    return best, [s[i] * r.get("scale", 1.0) for i in best]


def routed_ff(h, p, f):
    r = f["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        best, weights = choose(p["router"] @ h[t], p["correction"], r)
        for i, w in zip(best, weights):
            if i >= r["experts"]:
                out[t] += w * h[t]
            else:
                out[t] += w * gated_ff(h[t], p[f"e{i}.gate"], p[f"e{i}.up"], p[f"e{i}.down"])
    if f.get("shared"):
        gate = 1.0 / (1.0 + torch.exp(-(h @ p["shared.sg"].T)))
        out = out + gate * gated_ff(h, p["shared.gate"], p["shared.up"], p["shared.down"])
    return out


def feed_forward(h, p, f):
    return gated_ff(h, p["gate"], p["up"], p["down"]) if f["kind"] == "dense" else routed_ff(h, p, f)


# --------------------------------------------------------------------------------------------- the model
def sub(tensors, prefix):
    return {n[len(prefix):]: t for n, t in tensors.items() if n.startswith(prefix)}


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, tensors, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token (float64), and, asked for, the sum of the streams after
    every layer."""
    tensors = {n: t.to(F64) for n, t in tensors.items()}
    eps, n_streams = cfg["norm"]["eps"], cfg.get("streams")
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x0 = tensors["embed"][ids] + tensors["pos"][: len(ids)]
    xs = [x0.clone() for _ in range(n_streams or 1)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        t = sub(tensors, f"l{owner(cfg, i)}.")
        steps = [(1, lambda h: parallel_mixer(h, sub(t, "mix."), layer["mixer"], eps))]
        if layer.get("mlp") is not None:
            steps.append((2, lambda h: feed_forward(h, sub(t, "mlp."), layer["mlp"])))
        for n, fn in steps:
            if n_streams is None:
                xs[0] = xs[0] + fn(rmsnorm(xs[0], 1.0 + t[f"norm{n}"], eps))
                continue
            read, write, mix = t[f"hc{n}.in"], t[f"hc{n}.out"], t[f"hc{n}.mix"]
            y = fn(rmsnorm(sum(read[s] * xs[s] for s in range(n_streams)), 1.0 + t[f"norm{n}"], eps))
            xs = [sum(mix[s, d] * xs[s] for s in range(n_streams)) + write[d] * y for d in range(n_streams)]
        after.append(sum(xs))
    logits = rmsnorm(sum(xs), 1.0 + tensors["final.norm"], eps) @ tensors["embed"].T
    return (logits, torch.stack(after)) if return_layers else logits

"""Plain statement of the Barotar decoder, one function per mechanism, token loops where the equations have them.

Nothing here is fast and nothing is shared with the package: the tests hold the framework's kernels, caches and
schedules against these functions. Weights come as a dict of tensors under the checkpoint's names; every function works
in the dtype it is given (the tests use float64).
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return torch.where(x >= 0, 1 / (1 + torch.exp(-x.clamp_min(0))), torch.exp(x.clamp_max(0)) / (1 + torch.exp(x.clamp_max(0))))


def silu(x):
    return x * sigmoid(x)


def gelu(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


# ---- linear attention with a decay per key channel ----------------------------------------------------------------
def gla_decay(z, tau):
    return sigmoid(z) ** (1.0 / tau)


def rwkv_decay(z):
    return torch.exp(-torch.exp(z))


def gla_rule(q, k, v, alpha, S):
    """q, k, alpha [T, H, dk], v [T, H, dv], S [H, dk, dv] -> (o [T, H, dv], S after the last token)."""
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out, S


def rwkv_rule(r, k, v, w, u, S):
    """As above with a read before the update and `u` [H, dk] weighing the current token in that read."""
    out = torch.zeros_like(v)
    for t in range(r.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return out, S


def gla(w, p, m, h, state, eps):
    H, dk, dv, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = (h @ w[p + "q"].t()).reshape(T, H, dk) / math.sqrt(dk)
    k = (h @ w[p + "k"].t()).reshape(T, H, dk)
    v = (h @ w[p + "v"].t()).reshape(T, H, dv)
    z = ((h @ w[p + "a1"].t()) @ w[p + "a2"].t() + w[p + "a2.b"]).reshape(T, H, dk)
    if not state:
        state["S"] = torch.zeros(H, dk, dv, dtype=h.dtype)
    o, state["S"] = gla_rule(q, k, v, gla_decay(z, m["tau"]), state["S"])
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * dv)
    return (o * silu(h @ w[p + "g"].t())) @ w[p + "o"].t()


# ---- attention in a window, with a sink and capped scores -------------------------------------------------------------
def rotate(x, positions, dims, base):
    """x [T, H, d]: the pairs (2i, 2i + 1) of the first `dims` columns turned by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def window_attend(q, k, v, scale, cap, size, sink):
    """q [T, H, d] of the last T positions, k [L, G, d] / v [L, G, e] of all; a row at a time."""
    T, H, L = q.shape[0], q.shape[1], k.shape[0]
    of = torch.arange(H) // (H // k.shape[1])                # the key head of every query head
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        i = L - T + t
        lo = max(0, i - size + 1)
        s = cap * torch.tanh(torch.einsum("hd,lhd->hl", q[t], k[lo:i + 1, of]) * scale / cap)
        top = torch.maximum(s.max(-1).values, sink)
        e = torch.exp(s - top[:, None])
        out[t] = torch.einsum("hl,lhe->he", e / (e.sum(-1) + torch.exp(sink - top))[:, None], v[lo:i + 1, of])
    return out


def window_attention(w, p, m, h, positions, state, eps):
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q = rms((h @ w[p + "q"].t()).reshape(T, H, d), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].t()).reshape(T, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].t()).reshape(T, G, e)
    q, k = (rotate(x, positions, m["rot"]["dims"], m["rot"]["base"]) for x in (q, k))
    state["k"] = k = torch.cat([state["k"], k]) if state else k
    state["v"] = v = torch.cat([state["v"], v]) if "v" in state else v
    o = window_attend(q, k, v, m["scale"], m["softcap"], m["mask"]["size"], w[p + "sink"])
    return o.reshape(T, H * e) @ w[p + "o"].t()


def shifted(h, last, mu):
    """Every row moved towards the row before it (`last` before the first) by mu per column."""
    before = torch.cat([last[None], h[:-1]])
    return h + (before - h) * mu


def rwkv(w, p, m, h, state, eps):
    H, d, T = m["heads"], m["dim"], h.shape[0]
    if not state:
        state["h"], state["S"] = torch.zeros(h.shape[1], dtype=h.dtype), torch.zeros(H, d, d, dtype=h.dtype)
    mix = {s: shifted(h, state["h"], w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].t()).reshape(T, H, d) for s in "rkv")
    z = torch.tanh(mix["w"] @ w[p + "w1"].t()) @ w[p + "w2"].t() + w[p + "w0"]
    o, state["S"] = rwkv_rule(r, k, v, rwkv_decay(z).reshape(T, H, d), w[p + "u"], state["S"])
    state["h"] = h[-1]
    o = rms(o, eps).reshape(T, H * d) * w[p + "norm"]
    return (o * silu(mix["g"] @ w[p + "g"].t())) @ w[p + "o"].t()


def parallel(w, p, m, h, positions, state, eps):
    left, right = state.setdefault("left", {}), state.setdefault("right", {})
    return m["left_scale"] * window_attention(w, p + "left.", m["left"], h, positions, left, eps) \
        + m["right_scale"] * rwkv(w, p + "right.", m["right"], h, right, eps)


# ---- feed-forward ---------------------------------------------------------------------------------------------------
def geglu(w, p, h):
    return (gelu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def clamped_glu(w, p, h, limit):
    g = torch.clamp(h @ w[p + "gate"].t(), max=limit)
    u = torch.clamp(h @ w[p + "up"].t(), -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].t()


def route(logits, top, groups, keep):
    """-> per token a list of (expert, weight): sigmoid scores, the best `keep` of equal neighbouring groups by the sum of
    their two largest, then the `top` largest inside those; the weight is the score itself."""
    out = []
    for s in sigmoid(logits):
        n = len(s) // groups
        best = [float(sum(sorted(s[g * n:(g + 1) * n].tolist())[-2:])) for g in range(groups)]
        kept = sorted(range(groups), key=lambda g: (-best[g], g))[:keep]
        may = [e for g in sorted(kept) for e in range(g * n, (g + 1) * n)]
        out.append([(e, s[e]) for e in sorted(may, key=lambda e: (-float(s[e]), e))[:top]])
    return out


def experts(w, p, m, h):
    r, out = m["router"], torch.zeros_like(h)
    for t, chosen in enumerate(route(h @ w[p + "router"].t(), r["top"], r["groups"]["count"], r["groups"]["keep"])):
        for e, weight in chosen:
            out[t] += weight * clamped_glu(w, p + f"e{e}.", h[t:t + 1], m["expert"]["limit"])[0]
    return out


class Model:
    """Feeds tokens of one sequence at a time: `forward(ids, cache)` -> logits [T, vocab]; `cache` from `new_cache()`."""

    def __init__(self, config: dict, weights: dict, dtype=torch.float64):
        self.c, self.w = config, {k: v.to(dtype) for k, v in weights.items()}

    def new_cache(self):
        return {"length": 0, "layers": [{} for _ in self.c["layers"]]}

    @torch.no_grad()
    def forward(self, ids, cache, layers_out=None):
        c, w, eps = self.c, self.w, self.c["norm"]["eps"]
        ids = torch.as_tensor(ids)
        pos = torch.arange(cache["length"], cache["length"] + len(ids))
        x = w["embed"][ids]
        for i, layer in enumerate(c["layers"]):
            l, st = f"l{i}.", cache["layers"][i]
            h = rms(x, eps) * w[l + "norm1"]
            if layer["type"] == "gla":
                y = gla(w, l + "mix.", layer["mixer"], h, st, eps)
            else:
                y = parallel(w, l + "mix.", layer["mixer"], h, pos, st, eps)
            x = x + rms(y, eps) * w[l + "norm1b"]
            m = layer["mlp"]
            if m is not None:
                h = rms(x, eps) * w[l + "norm2"]
                y = geglu(w, l + "mlp.", h) if m["kind"] == "dense" else experts(w, l + "mlp.", m, h)
                x = x + rms(y, eps) * w[l + "norm2b"]
            if layers_out is not None:
                layers_out.append(x)
        cache["length"] += len(ids)
        return (rms(x, eps) * w["final.norm"]) @ w["embed"].t()

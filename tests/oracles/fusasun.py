"""Plain statement of the Fusasun decoder, one function per mechanism, token loops where the equations have them.

Nothing here is fast and nothing is shared with the package: the tests hold the framework's kernels, caches and
schedules against these functions. Weights come as a dict of tensors under the checkpoint's names; every function works
in the dtype it is given (the tests use float64).
"""
from __future__ import annotations

import math

import torch

from .barotar import rms, sigmoid, silu


# ---- positions --------------------------------------------------------------------------------------------------------
def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_frequencies(dims, base, s):
    """Short wavelengths stay, long ones are stretched by `factor`, those between go over from one to the other."""
    out = []
    for f in plain_frequencies(dims, base):
        wave = 2 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            u = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - u) * f / s["factor"] + u * f)
    return out


def yarn_frequencies(dims, base, s):
    """-> frequencies, and what cos and sin are multiplied by."""
    at = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, positions, frequencies, size=1.0):
    """x [T, H, d]: columns 2i and 2i + 1 turned by position * frequency i; columns behind the last pair pass. `size` multiplies
    cos and sin."""
    out = x.clone()
    for i, f in enumerate(frequencies):
        a = positions.to(x.dtype) * f
        c, s = size * torch.cos(a)[:, None], size * torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---- the residual -----------------------------------------------------------------------------------------------------
def gated_sum(x, y, h, w, b, w_post, eps):
    """x + rms(y * sigmoid(W h + b)) w_post."""
    return x + rms(y * sigmoid(h @ w.t() + b), eps) * w_post


def input_conv(w, h, state):
    """h + a causal convolution of it, channel by channel; `state["h"]`: the last inputs."""
    taps = w.shape[1]
    past = state.get("h", torch.zeros(taps - 1, h.shape[1], dtype=h.dtype))
    both = torch.cat([past, h])
    state["h"] = both[both.shape[0] - (taps - 1):]
    out = h.clone()
    for t in range(h.shape[0]):
        for j in range(taps):
            out[t] += w[:, j] * both[t + j]
    return out


# ---- attention --------------------------------------------------------------------------------------------------------
def softmax_sum(q, k, v, scale):
    """q [H, d] over k [n, H, d], v [n, H, e]."""
    s = torch.einsum("hd,nhd->hn", q, k) * scale
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return torch.einsum("hn,nhe->he", e / e.sum(-1, keepdim=True), v)


def window(q, k, v, scale, size):
    """q [T, H, d] of the last T positions over the `size` latest of k [L, H, d], v [L, H, e]."""
    L, T = k.shape[0], q.shape[0]
    out = torch.zeros(T, q.shape[1], v.shape[2], dtype=q.dtype)
    for t in range(T):
        i = L - T + t
        lo = max(0, i - size + 1)
        out[t] = softmax_sum(q[t], k[lo:i + 1], v[lo:i + 1], scale)
    return out


def pooled_window(q, k, v, scale, size, pool):
    """As `window`, and before it the mean key and value of every block of `pool` tokens that ends before the window."""
    L, T = k.shape[0], q.shape[0]
    out = torch.zeros(T, q.shape[1], v.shape[2], dtype=q.dtype)
    blocks = L // pool
    mk = k[:blocks * pool].reshape(blocks, pool, *k.shape[1:]).mean(1)
    mv = v[:blocks * pool].reshape(blocks, pool, *v.shape[1:]).mean(1)
    for t in range(T):
        i = L - T + t
        seen = [j for j in range(L) if 0 <= i - j < size]
        past = [b for b in range(blocks) if b * pool + pool - 1 <= i - size]
        out[t] = softmax_sum(q[t], torch.cat([mk[past], k[seen]]), torch.cat([mv[past], v[seen]]), scale)
    return out


def heads_of(x, H):
    """Every query head's own copy of its key head's rows."""
    return x[:, torch.arange(H) // (H // x.shape[1])]


def attention(w, p, m, h, positions, state, eps):
    H, G, d, e, T, r = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0], m["rot"]
    turn = lambda x: rotate(x, positions, banded_frequencies(r["dims"], r["base"], r["scaling"]))
    q = turn((h @ w[p + "q"].t()).reshape(T, H, d))
    k = turn((h @ w[p + "k"].t()).reshape(T, G, d))
    v = (h @ w[p + "v"].t()).reshape(T, G, e)
    state["k"] = k = torch.cat([state["k"], k]) if "k" in state else k
    state["v"] = v = torch.cat([state["v"], v]) if "v" in state else v
    o = pooled_window(q, heads_of(k, H), heads_of(v, H), m["scale"], m["mask"]["size"], m["mask"]["pool"])
    return o.reshape(T, H * e) @ w[p + "o"].t()


def latent_attention(w, p, m, h, positions, state, eps):
    """Keys and values made from a small latent row per token, one rotated key part for all heads, queries through a latent, a
    gate per head."""
    H, d, r, e, L, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    q = ((rms(h @ w[p + "dq"].t(), eps) * w[p + "dq.norm"]) @ w[p + "uq"].t()).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].t()
    c = rms(down[:, :L], eps) * w[p + "dkv.norm"]
    f, size = yarn_frequencies(r, m["rot"]["base"], m["rot"]["scaling"])
    turn = lambda x: rotate(x, positions, f, size)
    kr = turn(down[:, None, L:])
    state["c"] = c = torch.cat([state["c"], c]) if "c" in state else c
    state["r"] = kr = torch.cat([state["r"], kr]) if "r" in state else kr
    N = c.shape[0]
    k = torch.cat([(c @ w[p + "uk"].t()).reshape(N, H, d), kr.expand(N, H, r)], -1)
    v = (c @ w[p + "uv"].t()).reshape(N, H, e)
    q = torch.cat([q[..., :d], turn(q[..., d:])], -1)
    o = window(q, k, v, m["scale"], m["mask"]["size"]) * sigmoid(h @ w[p + "g"].t())[..., None]
    return o.reshape(T, H * e) @ w[p + "o"].t()


# ---- feed-forward -----------------------------------------------------------------------------------------------------
def swiglu(w, p, h):
    return (silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def experts(w, p, f, h, ids, table):
    """Each token's experts stand in the table's row of its id; all weigh the same."""
    top, out = f["router"]["top"], torch.zeros_like(h)
    for t, token in enumerate(ids.tolist()):
        for e in table[token].tolist():
            out[t] += swiglu(w, f"{p}e{e}.", h[t:t + 1])[0] / top
    return out


class Model:
    """Feeds tokens of one sequence at a time: `forward(ids, cache)` -> logits [T, vocab]; `cache` from `new_cache()`."""

    def __init__(self, config: dict, weights: dict, dtype=torch.float64):
        self.c = config
        self.tables = {k: v for k, v in weights.items() if k.endswith(".table")}
        self.w = {k: v.to(dtype) for k, v in weights.items() if k not in self.tables}

    def new_cache(self):
        return {"length": 0, "layers": [{} for _ in self.c["layers"]]}

    @torch.no_grad()
    def forward(self, ids, cache, layers_out=None):
        c, w, eps = self.c, self.w, self.c["norm"]["eps"]
        ids = torch.as_tensor(ids)
        pos = torch.arange(cache["length"], cache["length"] + len(ids))
        x = w["embed"][ids] * c["embedding"]["scale"]
        mixers = {"attention": attention, "latent_attention": latent_attention}
        for i, layer in enumerate(c["layers"]):
            l, st, f = f"l{i}.", cache["layers"][i], layer["mlp"]
            h = rms(x, eps) * w[l + "norm1"]
            y = mixers[layer["type"]](w, l + "mix.", layer["mixer"], input_conv(w[l + "canon1"], h, st), pos, st, eps)
            x = gated_sum(x, y, h, w[l + "rg1"], w[l + "rg1.b"], w[l + "norm1b"], eps)
            if f is not None:
                h = rms(x, eps) * w[l + "norm2"]
                y = experts(w, l + "mlp.", f, h, ids, self.tables[l + "mlp.table"])
                x = gated_sum(x, y, h, w[l + "rg2"], w[l + "rg2.b"], w[l + "norm2b"], eps)
            if layers_out is not None:
                layers_out.append(x)
        cache["length"] += len(ids)
        return (rms(x, eps) * w["final.norm"]) @ w["head"].t()

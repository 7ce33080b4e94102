"""Plain statement of the Diderax decoder, one function per mechanism, token loops where the equations have them.

Nothing here is fast and nothing is shared with the package: the tests hold the framework's kernels, caches and
schedules against these functions. Weights come as a dict of tensors under the checkpoint's names; every function works
in the dtype it is given (the tests use float64).
"""
from __future__ import annotations

import torch

from .barotar import gla, rms, sigmoid, silu


# ---- positions --------------------------------------------------------------------------------------------------------
def rotate(x, positions, dims, base, factor=1.0):
    """x [T, H, d]: columns i and i + dims / 2 of the first `dims` turned by position * base^(-2i / dims) / factor."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        a = positions.to(x.dtype) * base ** (-2.0 * i / dims) / factor
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


# ---- softmax attention with a sink ------------------------------------------------------------------------------------
def attend(q, k, v, scale, sink):
    """q [T, H, d] of the last T positions, k [L, G, d] / v [L, G, e] of all, sink [H]: one more score in every denominator."""
    T, H, L = q.shape[0], q.shape[1], k.shape[0]
    of = torch.arange(H) // (H // k.shape[1])                # the key head of every query head
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        n = L - T + t + 1
        s = torch.einsum("hd,lhd->hl", q[t], k[:n, of]) * scale
        top = torch.maximum(s.max(-1).values, sink)
        e = torch.exp(s - top[:, None])
        out[t] = torch.einsum("hl,lhe->he", e / (e.sum(-1) + torch.exp(sink - top))[:, None], v[:n, of])
    return out


def attention(w, p, m, h, positions, state, eps):
    """Keys that are values too (as projected), norms over whole projections, a sink of score 0, an output gate."""
    H, G, d, T = m["heads"], m["kv_heads"], m["dim"], h.shape[0]
    q, k = h @ w[p + "q"].t(), h @ w[p + "k"].t()
    v = k.reshape(T, G, d)
    q = (rms(q, eps) * w[p + "q.norm"]).reshape(T, H, d)
    k = (rms(k, eps) * w[p + "k.norm"]).reshape(T, G, d)
    r = m["rot"]
    q, k = (rotate(x, positions, r["dims"], r["base"], r["scaling"]["factor"]) for x in (q, k))
    state["k"] = k = torch.cat([state["k"], k]) if state else k
    state["v"] = v = torch.cat([state["v"], v]) if "v" in state else v
    o = attend(q, k, v, m["scale"], torch.zeros(H, dtype=h.dtype)).reshape(T, H * d)
    return (o * sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


def latent_attention(w, p, m, h, positions, state, eps):
    """Keys and values made from a small latent row per token, one rotated key part for all heads, queries through a latent."""
    H, d, r, e, L, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    q = ((rms(h @ w[p + "dq"].t(), eps) * w[p + "dq.norm"]) @ w[p + "uq"].t()).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].t()
    c = rms(down[:, :L], eps) * w[p + "dkv.norm"]
    turn = lambda x: rotate(x, positions, r, m["rot"]["base"])
    kr = turn(down[:, None, L:])
    state["c"] = c = torch.cat([state["c"], c]) if state else c
    state["r"] = kr = torch.cat([state["r"], kr]) if "r" in state else kr
    N = c.shape[0]
    k = torch.cat([(c @ w[p + "uk"].t()).reshape(N, H, d), kr.expand(N, H, r)], -1)
    v = (c @ w[p + "uv"].t()).reshape(N, H, e)
    q = torch.cat([q[..., :d], turn(q[..., d:])], -1)
    return attend(q, k, v, m["scale"], w[p + "sink"]).reshape(T, H * e) @ w[p + "o"].t()


# ---- feed-forward -----------------------------------------------------------------------------------------------------
def swiglu(w, p, h):
    return (silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def swiglu_biased(w, p, h):
    a = silu(h @ w[p + "gate"].t() + w[p + "gate.b"]) * (h @ w[p + "up"].t() + w[p + "up.b"])
    return a @ w[p + "down"].t() + w[p + "down.b"]


def route(logits, correction, top, groups, keep, scale):
    """-> per token a list of (expert, weight). Softmax scores s; choices by s + correction, only inside the `keep` neighbouring
    groups whose largest choices are largest; weights s over their sum, times `scale`."""
    out = []
    for z in logits:
        s = torch.exp(z - z.max())
        s = s / s.sum()
        c, n = s + correction, len(s) // groups
        best = [float(c[g * n:(g + 1) * n].max()) for g in range(groups)]
        kept = sorted(range(groups), key=lambda g: (-best[g], g))[:keep]
        may = [e for g in sorted(kept) for e in range(g * n, (g + 1) * n)]
        chosen = sorted(may, key=lambda e: (-float(c[e]), e))[:top]
        total = sum(s[e] for e in chosen) + 1e-20
        out.append([(e, s[e] / total * scale) for e in chosen])
    return out


def experts(w, p, m, h):
    """Routed experts, of which the last `identity` hand the row back, and the shared one behind its gate."""
    r, out = m["router"], torch.zeros_like(h)
    groups = r["groups"]
    for t, chosen in enumerate(route(h @ w[p + "router"].t(), w[p + "correction"], r["top"], groups["count"], groups["keep"], r["scale"])):
        for e, weight in chosen:
            out[t] += weight * (swiglu(w, p + f"e{e}.", h[t:t + 1])[0] if e < r["experts"] else h[t])
    return out + swiglu(w, p + "shared.", h) * sigmoid(h @ w[p + "shared.sg"].t())


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
            l, m, st = f"l{i}.", layer["mixer"], cache["layers"][i]
            h = rms(x, eps) * w[l + "norm1"]
            if layer["type"] == "gla":
                y = gla(w, l + "mix.", m, h, st, eps)
            else:
                y = {"attention": attention, "latent_attention": latent_attention}[layer["type"]](w, l + "mix.", m, h, pos, st, eps)
            x = x + w[l + "ls1"] * y
            f = layer["mlp"]
            if f is not None:
                h = rms(x, eps) * w[l + "norm2"]
                y = swiglu_biased(w, l + "mlp.", h) if f["kind"] == "dense" else experts(w, l + "mlp.", f, h)
                x = x + w[l + "ls2"] * y
            if layers_out is not None:
                layers_out.append(x)
        cache["length"] += len(ids)
        return (rms(x, eps) * w["final.norm"]) @ w["head"].t()

"""Plain statement of the Gafapel decoder, one function per mechanism, token loops where the equations have them.

Nothing here is fast and nothing is shared with the package: the tests hold the framework's kernels, caches and
schedules against these functions. Weights come as a dict of tensors under the checkpoint's names; every function works
in the dtype it is given (the tests use float64).
"""
from __future__ import annotations

import torch


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def embed(w, ids, positions, eps):
    return rms(w["embed"][ids] + w["pos"][positions], eps) * w["embed.norm"]


def hyper_in(x, w_in):
    """x [T, S, D] -> the sublayer's input before its norm."""
    return torch.einsum("tsd,s->td", x, w_in)


def hyper_out(x, y, mix, out):
    """Every stream from the old ones (mix[from, to]) plus its share of the sublayer's output."""
    return torch.einsum("tsd,sr->trd", x, mix) + out[None, :, None] * y[:, None, :]


def short_conv(u, hist, taps, bias):
    """u [T, C], hist [K-1, C] the inputs before it -> (silu of the causal convolution, the new history)."""
    k = taps.shape[1]
    full = torch.cat([hist, u], 0)
    rows = []
    for t in range(u.shape[0]):
        acc = bias.clone()
        for j in range(k):
            acc = acc + taps[:, j] * full[t + j]
        rows.append(acc)
    return silu(torch.stack(rows)), full[full.shape[0] - (k - 1):]


def state_space(x, B, C, dt, A_log, dt_bias, D, S, groups):
    """x [T, H, P], B / C [T, G, N], dt [T, H] raw, S [H, N, P] -> (y [T, H, P], S after the last token)."""
    T, heads, _ = x.shape
    step = softplus(dt + dt_bias)
    out = torch.zeros_like(x)
    S = S.clone()
    per = heads // groups
    for t in range(T):
        for h in range(heads):
            g = h // per
            S[h] = torch.exp(-torch.exp(A_log[h]) * step[t, h]) * S[h] + step[t, h] * torch.outer(B[t, g], x[t, h])
            out[t, h] = S[h].t() @ C[t, g] + D[h] * x[t, h]
    return out, S


def gated_group_norm(y, z, weight, parts, eps):
    g = y * silu(z)
    return rms(g.reshape(g.shape[0], parts, -1), eps).reshape(g.shape) * weight


def mamba2(w, p, m, h, state, eps):
    """One Mamba-2 mixer over h [T, D]; `state` = {"hist", "S"} or empty, updated in place."""
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, T = H * P, h.shape[0]
    proj = h @ w[p + "in"].t()
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    if not state:
        state["hist"] = torch.zeros(m["conv"] - 1, inner + 2 * G * N, dtype=h.dtype)
        state["S"] = torch.zeros(H, N, P, dtype=h.dtype)
    xbc, state["hist"] = short_conv(xbc, state["hist"], w[p + "conv"], w[p + "conv.b"])
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    y, state["S"] = state_space(x, B, C, dt, w[p + "A_log"], w[p + "dt_bias"], w[p + "D"], state["S"], G)
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].t()


def attend(q, k, v, scale):
    """q [T, H, d] of the last T positions, k / v of all positions: causal softmax attention, a row at a time."""
    T, L = q.shape[0], k.shape[0]
    out = torch.zeros(T, q.shape[1], v.shape[2], dtype=q.dtype)
    for t in range(T):
        n = L - T + t + 1
        s = torch.einsum("hd,lhd->hl", q[t], k[:n]) * scale
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[t] = torch.einsum("hl,lhv->hv", e / e.sum(-1, keepdim=True), v[:n])
    return out


def latent_attention(w, p, m, h, state, eps):
    """Attention over keys and values expanded from the cached latents; `state` = {"c"} or empty."""
    H, d, v, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = (h @ w[p + "q"].t()).reshape(T, H, d)
    c = rms(h @ w[p + "dkv"].t(), eps) * w[p + "dkv.norm"]
    state["c"] = c = torch.cat([state["c"], c], 0) if state else c
    out = attend(q, (c @ w[p + "uk"].t()).reshape(-1, H, d), (c @ w[p + "uv"].t()).reshape(-1, H, v), m["scale"])
    gate = 1 / (1 + torch.exp(-(h @ w[p + "g"].t())))
    return (out.reshape(T, H * v) * gate) @ w[p + "o"].t()


def glu(w, p, h):
    return (silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def route(logits, top):
    """-> per token a list of (expert, weight): the largest logits, weighed by the softmax over them."""
    out = []
    for z in logits:
        order = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[:top]
        e = torch.exp(z[order] - z[order].max())
        out.append([(i, x) for i, x in zip(order, e / e.sum())])
    return out


def experts(w, p, m, h):
    out = torch.zeros_like(h)
    for t, chosen in enumerate(route(h @ w[p + "router"].t() + w[p + "router.b"], m["router"]["top"])):
        for e, weight in chosen:
            out[t] += weight * glu(w, p + f"e{e}.", h[t:t + 1])[0]
    return out


MIXERS = {"mamba2": mamba2, "mamba2_2": mamba2, "latent_attention": latent_attention}


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
        x = embed(w, ids, pos, eps)[:, None, :].repeat(1, c["streams"], 1)
        for i, layer in enumerate(c["layers"]):
            l = f"l{i}."
            u = rms(hyper_in(x, w[l + "hc1.in"]), eps) * w[l + "norm1"]
            y = MIXERS[layer["type"]](w, l + "mix.", layer["mixer"], u, cache["layers"][i], eps)
            x = hyper_out(x, y, w[l + "hc1.mix"], w[l + "hc1.out"])
            m = layer["mlp"]
            if m is not None:
                u = rms(hyper_in(x, w[l + "hc2.in"]), eps) * w[l + "norm2"]
                y = glu(w, l + "mlp.", u) if m["kind"] == "dense" else experts(w, l + "mlp.", m, u)
                x = hyper_out(x, y, w[l + "hc2.mix"], w[l + "hc2.out"])
            if layers_out is not None:
                layers_out.append(x.sum(1))
        cache["length"] += len(ids)
        return (rms(x.sum(1), eps) * w["final.norm"]) @ w["head"].t()

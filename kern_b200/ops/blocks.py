"""CPU statements of the kernels in hyper.cu, resid.cu, linear.cu, ssd.cu, lin_attn.cu, latent.cu, attn_window.cu, conv_add.cu (and the forms
of the same mechanisms in mla_decode.cu / moe.cu / ssd_chunk.cu / lin_attn_chunk.cu / attn_fmha.cu / gemm_bf16.cu):
what each launch computes, over the same arguments, for `kern_b200.cpu.CpuRuntime`. Rounding follows the buffers' types."""
from __future__ import annotations

import torch
import torch.nn.functional as F

from ..cpu import CPU_KERNELS, _rows_of

T = torch.Tensor


def _f(t):
    return t.float()


def _rows(t, n, cols, stride):
    """[n, cols] view of a flat buffer whose rows are `stride` apart, from the buffer's own start."""
    return torch.as_strided(t, (n, cols), (stride, 1))


def _norm(u, w, eps):
    return u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps) * _f(w)


# ---- hyper-connections ----
def k_hyper_embed(g, ids, positions, table, pos_table, w_embed, w_in, w_norm, x, xn, d, s, vocab, max_pos, eps, err):
    n = g[0]
    tok, pos = ids[:n].long(), positions[:n].long()
    if ((tok < 0) | (tok >= vocab) | (pos < 0) | (pos >= max_pos)).any():
        err[0] = 300
    e = _f(table[: vocab * d].view(vocab, d)[tok.clamp(0, vocab - 1)]) + _f(pos_table[: max_pos * d].view(max_pos, d)[pos.clamp(0, max_pos - 1)])
    e = _norm(e, w_embed[:d], eps)
    x[: n * s * d] = e[:, None].expand(n, s, d).reshape(-1)
    xn[: n * d] = _norm(e * _f(w_in[:s]).sum(), w_norm[:d], eps).to(xn.dtype).reshape(-1)


def _mixed(n, x, y, perm, topw, w_mix, w_out, d, s, k):
    xs = x[: n * s * d].view(n, s, d)
    if isinstance(perm, T):
        rows = _f(y[: n * k * d].view(-1, d)[perm[: n * k].long()]).view(n, k, d)
        yv = (rows * topw[: n * k].view(n, k, 1)).sum(1)
    else:
        yv = _f(y[: n * d].view(n, d))
    return torch.einsum("tsd,sr->trd", xs, _f(w_mix[: s * s].view(s, s))) + _f(w_out[:s])[None, :, None] * yv[:, None]


def k_hyper_mix(g, x, y, perm, topw, w_mix, w_out, w_in, w_norm, xn, d, s, k, eps):
    n = g[0]
    new = _mixed(n, x, y, perm, topw, w_mix, w_out, d, s, k)
    x[: n * s * d] = new.reshape(-1)
    xn[: n * d] = _norm(torch.einsum("tsd,s->td", new, _f(w_in[:s])), w_norm[:d], eps).to(xn.dtype).reshape(-1)


def k_hyper_last(g, x, y, perm, topw, w_mix, w_out, hidden, d, s, k):
    n = g[0]
    hidden[: n * d] = _mixed(n, x, y, perm, topw, w_mix, w_out, d, s, k).sum(1).reshape(-1)


def k_row_norm(g, src, cu, rows, w, y, src_rows, d, eps):
    n = g[0]
    at = cu[1:n + 1].long() - 1 if isinstance(cu, T) else (rows[:n].long() if isinstance(rows, T) else torch.arange(n))
    u = src[: src_rows * d].view(src_rows, d)[at.clamp(0, src_rows - 1)]
    y[: n * d] = _norm(u, w[:d], eps).to(y.dtype).reshape(-1)


# ---- the residual with norms on both sides ----
def k_resid_embed(g, ids, table, w, x, xn, d, vocab, scale, eps, err):
    n = g[0]
    tok = ids[:n].long()
    if ((tok < 0) | (tok >= vocab)).any():
        err[0] = 300
    e = _f(table[: vocab * d].view(vocab, d)[torch.where((tok < 0) | (tok >= vocab), 0, tok)]) * scale
    x[: n * d] = e.reshape(-1)
    xn[: n * d] = _norm(e, w[:d], eps).to(xn.dtype).reshape(-1)


def _routed_rows(n, y, perm, topw, d, k):
    if isinstance(perm, T):
        return (_f(y.view(-1)[: n * k * d].view(-1, d)[perm[: n * k].long()]).view(n, k, d) * topw[: n * k].view(n, k, 1)).sum(1)
    return _f(y[: n * d].view(n, d))


def _resid_out(n, x, v, w_next, xn, hidden, d, eps):
    new = x[: n * d].view(n, d) + v
    if isinstance(hidden, T):
        hidden[: n * d] = new.reshape(-1)
    else:
        x[: n * d] = new.reshape(-1)
        xn[: n * d] = _norm(new, w_next[:d], eps).to(xn.dtype).reshape(-1)


def k_resid_mix(g, x, y, perm, topw, w_post, w_next, xn, hidden, d, k, eps):
    v = _routed_rows(g[0], y, perm, topw, d, k)
    _resid_out(g[0], x, _norm(v, w_post[:d], eps) if isinstance(w_post, T) else v, w_next, xn, hidden, d, eps)


def k_resid_scale(g, x, y, perm, topw, shared, gate, bias, scale, w_next, xn, hidden, d, k, gs, eps):
    n = g[0]
    if isinstance(perm, T):
        p, w = perm[: n * k].view(n, k).long(), topw[: n * k].view(n, k, 1)
        rows = _f(y.view(-1)[: n * k * d].view(-1, d)[p.clamp_min(0)])
        own = _f(xn[: n * d].view(n, 1, d)) if isinstance(xn, T) else torch.zeros(n, 1, d)
        v = (torch.where((p < 0)[..., None], own, rows) * w).sum(1)
    else:
        v = _f(y[: n * d].view(n, d))
    if isinstance(shared, T):
        v = v + torch.sigmoid(_rows(gate, n, 1, gs)) * _f(shared[: n * d].view(n, d))
    if isinstance(bias, T):
        v = v + _f(bias[:d])
    new = x[: n * d].view(n, d) + v * _f(scale[:d])
    if isinstance(hidden, T):
        hidden[: n * d] = new.reshape(-1)
    else:
        x[: n * d] = new.reshape(-1)
        xn[: n * d] = _norm(new, w_next[:d], eps).to(xn.dtype).reshape(-1)


# ---- matrix products ----
def _glu(v, kind, limit=0.0):
    g, u = v[:, :v.shape[1] // 2], v[:, v.shape[1] // 2:]
    if kind == "geglu":
        return F.gelu(g, approximate="tanh") * u
    if kind == "clamped":
        g = g.clamp(max=limit)
        return g * torch.sigmoid(1.702 * g) * (u.clamp(-limit, limit) + 1)
    return F.silu(g) * u


def _k_linear(glu):
    def run(g, a, w, c, m, n, k, lda, ldc, wsn, wsk, az, wz, cz, err, limit, bias):
        if m > g[1] * 64:
            err[0] = 300
        for z in range(g[2]):
            A = _f(_rows(a[z * az:], m, k, lda))
            W = _f(torch.as_strided(w[z * wz:], ((2 if glu else 1) * n, k), (wsn, wsk)))
            v = A @ W.t()
            if isinstance(bias, T):
                v = v + _f(bias[: v.shape[1]])
            _rows(c[z * cz:], m, n, ldc).copy_(_glu(v, glu, limit) if glu else v)
    return run


def k_gemm_heads(g, a, w, c, m, n, k, ldc, heads, err):
    lda = a._row_stride
    for h in range(heads):
        W = _f(w[h * n * k:(h + 1) * n * k].view(n, k))
        _rows(c[h * n:], m, n, ldc).copy_(_f(_rows(a[h * k:], m, k, lda)) @ W.t())


def _k_grouped(glu):
    def run(g, a, w, c, tiles, count, rows, n, k, wz, err, limit):
        for e, r0, nr, _ in tiles.view(-1, 4)[: int(count[0])].tolist():
            W = _f(w[e * wz: e * wz + (2 if glu else 1) * n * k].view(-1, k))
            v = _f(a[r0 * k:(r0 + nr) * k].view(nr, k)) @ W.t()
            c[r0 * n:(r0 + nr) * n] = (_glu(v, glu, limit) if glu else v).to(c.dtype).reshape(-1)
    return run


def _k_moe_gemm(glu):
    def run(g, a, w, c, tiles, count, rows, n, k, ldc, err, limit=0.0):
        wz = n * k
        for e, r0, nr, _ in tiles.view(-1, 4)[: int(count[0])].tolist():
            v = _f(a[r0 * k:(r0 + nr) * k].view(nr, k)) @ _f(w[e * wz:(e + 1) * wz].view(n, k)).t()
            _rows(c[r0 * ldc:], nr, ldc, ldc).copy_(_glu(v, glu, limit))
    return run


def k_copy_cols(g, src, dst, cols, stride):
    _rows(dst, g[0], cols, stride).copy_(src[: g[0] * cols].view(g[0], cols))


def k_rows_scatter(g, x, perm, out, entries, k, d):
    p = perm[:entries].long()
    ok = p >= 0
    out.view(-1)[: entries * d].view(-1, d)[p[ok]] = x.view(-1)[: (entries // k) * d].view(-1, d)[torch.arange(entries)[ok] // k]


def k_gate_mul(g, x, gate, out, n, d, xs, gs, os_):
    _rows(out, n, d, os_).copy_(_f(_rows(x, n, d, xs)) * torch.sigmoid(_f(_rows(gate, n, d, gs))))


def k_transpose_heads(g, src, dst, r, c):
    h = g[2]
    dst[: h * r * c] = src[: h * r * c].view(h, r, c).transpose(1, 2).reshape(-1)


# ---- Mamba-2 ----
def _window(state, line, line_bytes, keep, ch, dt):
    return state[line * line_bytes: line * line_bytes + keep * ch * dt.itemsize].view(dt).view(keep, ch)


def k_ssd_conv(g, x, y, state, lines, cu, w, bias, seqs, rows, ch, taps, xs, line_bytes):
    wt = _f(w[: ch * taps].view(ch, taps))
    for s in range(seqs):
        r0, r1 = _rows_of(cu, s)
        if r1 <= r0:
            continue
        ln = int(lines[s])
        hist = _f(_window(state, ln, line_bytes, taps - 1, ch, x.dtype)) if ln > 0 else torch.zeros(taps - 1, ch)
        full = torch.cat([hist, _f(_rows(x[r0 * xs:], r1 - r0, ch, xs))], 0)
        out = sum(full[j:j + r1 - r0] * wt[:, j] for j in range(taps)) + _f(bias[:ch])
        y[r0 * ch: r1 * ch] = F.silu(out).to(y.dtype).reshape(-1)


def k_ssd_conv_state(g, x, state, lines, cu, seqs, ch, taps, xs, line_bytes):
    for s in range(seqs):
        r0, r1 = _rows_of(cu, s)
        ln = int(lines[s])
        if r1 <= r0 or ln <= 0:
            continue
        win = _window(state, ln, line_bytes, taps - 1, ch, x.dtype)
        full = torch.cat([win, _rows(x[r0 * xs:], r1 - r0, ch, xs)], 0)
        win.copy_(full[full.shape[0] - (taps - 1):].clone())


def k_ssd_chunk(g, xbc, dt, y, state, lines, cu, A_log, dt_bias, D, seqs, H, P, N, G, dts, line_bytes, s_off, min_rows):
    k_ssd_rule(g, xbc, dt, y, state, lines, cu, A_log, dt_bias, D, seqs, H, P, N, G, dts, line_bytes, s_off, 0, 1 << 31, min_rows)


def k_ssd_rule(g, xbc, dt, y, state, lines, cu, A_log, dt_bias, D, seqs, H, P, N, G, dts, line_bytes, s_off, tb, max_rows, min_rows=1):
    inner, ch, rep = H * P, H * P + 2 * G * N, H // G
    for s in range(g[1]):
        r0, r1 = _rows_of(cu, s)
        n = r1 - r0
        if not min_rows <= n <= max_rows:
            continue
        ln = int(lines[s])
        Sb = state[ln * line_bytes + s_off: ln * line_bytes + s_off + H * P * N * 4].view(torch.float32).view(H, P, N)
        S = Sb.clone() if ln > 0 else torch.zeros(H, P, N)
        rows = _f(xbc[r0 * ch: r1 * ch].view(n, ch))
        x = rows[:, :inner].view(n, H, P)
        Bm = rows[:, inner:inner + G * N].view(n, G, N).repeat_interleave(rep, 1)
        Cm = rows[:, inner + G * N:].view(n, G, N).repeat_interleave(rep, 1)
        step = F.softplus(_f(_rows(dt[r0 * dts:], n, H, dts)) + _f(dt_bias[:H]), threshold=30)
        decay = torch.exp(-torch.exp(_f(A_log[:H])) * step)
        out = torch.empty(n, H, P)
        for t in range(n):
            S = decay[t][:, None, None] * S + step[t][:, None, None] * x[t][:, :, None] * Bm[t][:, None, :]
            out[t] = torch.einsum("hpn,hn->hp", S, Cm[t]) + _f(D[:H])[:, None] * x[t]
        y[r0 * inner: r1 * inner] = out.reshape(-1)
        if ln > 0:
            Sb.copy_(S)


def k_ssd_gate_norm(g, y, z, w, out, inner, parts, zs, eps):
    n = g[0]
    v = y[: n * inner].view(n, inner) * F.silu(_f(_rows(z, n, inner, zs)))
    v = v.view(n, parts, -1)
    v = (v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)).reshape(n, inner) * _f(w[:inner])
    out[: n * inner] = v.to(out.dtype).reshape(-1)


# ---- linear attention with a decay per key channel ----
def _kept(state, line, line_bytes, width):
    return state[line * line_bytes: line * line_bytes + width * 4].view(torch.float32)


def k_token_shift(g, h, mu, out, state, lines, cu, seqs, d, targets, line_bytes):
    m = _f(mu[: targets * d].view(targets, d))
    for s in range(seqs):
        r0, r1 = _rows_of(cu, s)
        if r1 <= r0:
            continue
        ln = int(lines[s])
        x = _f(h[r0 * d: r1 * d].view(-1, d))
        last = _kept(state, ln, line_bytes, d) if ln > 0 else torch.zeros(d)
        before = torch.cat([last[None], x[:-1]])
        out[r0 * targets * d: r1 * targets * d] = (x[:, None] + (before - x)[:, None] * m).to(out.dtype).reshape(-1)
        if not isinstance(cu, T) and ln > 0:
            last.copy_(x[-1])


def k_shift_state(g, h, state, lines, cu, seqs, d, line_bytes):
    for s in range(seqs):
        r0, r1 = _rows_of(cu, s)
        if r1 > r0 and int(lines[s]) > 0:
            _kept(state, int(lines[s]), line_bytes, d).copy_(_f(h[(r1 - 1) * d: r1 * d]))


def k_decay(g, a, w, bias, alpha, rows, n, rank, lda, mode, inv_tau):
    v = _f(_rows(a, rows, rank, lda))
    z = (torch.tanh(v) if mode else v) @ _f(w[: n * rank].view(n, rank)).t() + _f(bias[:n])
    alpha[: rows * n] = torch.exp(-torch.exp(z) if mode else F.logsigmoid(z) * inv_tau).reshape(-1)


def k_lin_rule(g, q, k, v, gate, alpha, u, norm, out, state, lines, cu, seqs, H, dk, dv, stride, norm_step, out_stride, line_bytes, s_off, fused,
               tb, max_rows, q_scale, out_scale, eps, min_rows=1):
    for s in range(seqs):
        r0, r1 = _rows_of(cu, s)
        n = r1 - r0
        if not min_rows <= n <= max_rows:
            continue
        ln = int(lines[s])
        Sb = state[ln * line_bytes + s_off: ln * line_bytes + s_off + H * dk * dv * 4].view(torch.float32).view(H, dk, dv)
        S = Sb.clone() if ln > 0 else torch.zeros(H, dk, dv)
        part = lambda t, c: _f(_rows(t[r0 * stride:], n, H * c, stride)).view(n, H, c)
        qq, kk, vv = part(q, dk) * q_scale, part(k, dk), part(v, dv)
        al, o = alpha[r0 * H * dk: r1 * H * dk].view(n, H, dk), torch.empty(n, H, dv)
        for t in range(n):
            kv = kk[t][:, :, None] * vv[t][:, None, :]
            if isinstance(u, T):
                o[t] = torch.einsum("hkv,hk->hv", S + _f(u[: H * dk].view(H, dk, 1)) * kv, qq[t])
            S = al[t][:, :, None] * S + kv
            if not isinstance(u, T):
                o[t] = torch.einsum("hkv,hk->hv", S, qq[t])
        if fused:
            k_lin_norm_gate((n,), o.reshape(-1), gate[r0 * stride:], norm, out[r0 * out_stride:], H, dv, stride, norm_step, out_stride, out_scale, eps)
        else:
            out[r0 * H * dv: r1 * H * dv] = o.reshape(-1)
        if ln > 0:
            Sb.copy_(S)


def k_lin_prep(g, q, k, alpha, u, prep, cu, seqs, H, dk, stride, min_rows, slots, q_scale):
    """The real buffer holds scaled and split factors; here the chunk kernel's statement is handed the arguments themselves."""
    prep._rows = (q, k, alpha, u, q_scale)


def k_lin_chunk(g, v, prep, out, state, lines, cu, seqs, H, dk, dv, stride, line_bytes, s_off, min_rows):
    q, k, alpha, u, q_scale = prep._rows
    k_lin_rule(g, q, k, v, 0, alpha, u, 0, out, state, lines, cu, seqs, H, dk, dv, stride, 0, 0, line_bytes, s_off, 0, 0, 1 << 31, q_scale, 1.0, 0.0, min_rows)


def k_lin_norm_gate(g, o, gate, w, out, H, dv, gs, norm_step, os_, out_scale, eps):
    n = g[0]
    x = o[: n * H * dv].view(n, H, dv)
    wt = _f(w[: H * dv].view(H, dv)) if norm_step else _f(w[:dv])
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * wt * out_scale
    _rows(out, n, H * dv, os_).copy_(y.reshape(n, -1) * F.silu(_f(_rows(gate, n, H * dv, gs))))


# ---- a convolution added to its input ----
def k_conv_add(g, h, out, state, lines, cu, w, seqs, rows, d, taps, line_bytes):
    wt = _f(w[: d * taps].view(d, taps))
    for s in range(seqs):
        r0, r1 = _rows_of(cu, s)
        if r1 <= r0:
            continue
        ln, n = int(lines[s]), r1 - r0
        past = _f(_window(state, ln, line_bytes, taps - 1, d, h.dtype)) if ln > 0 else torch.zeros(taps - 1, d)
        both = torch.cat([past, _f(h[r0 * d: r1 * d].view(n, d))])
        out[r0 * d: r1 * d] = (both[taps - 1:] + sum(wt[:, j] * both[j: j + n] for j in range(taps))).to(out.dtype).reshape(-1)
    k_ssd_conv_state(g, h, state, lines, cu, seqs, d, taps, d, line_bytes)


def _conv_rows(n, xn, w, out, state, lines, d, taps, line_bytes):
    k_conv_add(None, xn, out, state, lines, torch.arange(n + 1, dtype=torch.int32), w, n, n, d, taps, line_bytes)


def k_resid_embed_conv(g, ids, table, w_norm, x, xn, d, vocab, scale, eps, err, *conv):
    k_resid_embed(g, ids, table, w_norm, x, xn, d, vocab, scale, eps, err)
    w, out, state, lines, taps, line_bytes = conv
    _conv_rows(g[0], xn, w, out, state, lines, d, taps, line_bytes)


def k_resid_gate(g, x, y, perm, topw, w_post, w_next, xn, hidden, d, k, eps, gate, gate_b):
    n = g[0]
    v = _routed_rows(n, y, perm, topw, d, k) * torch.sigmoid(_f(gate[: n * d].view(n, d)) + _f(gate_b[:d]))
    _resid_out(n, x, _norm(v, w_post[:d], eps), w_next, xn, hidden, d, eps)


def k_resid_gate_conv(g, x, y, perm, topw, w_post, w_next, xn, d, k, eps, gate, gate_b, w, out, state, lines, taps, line_bytes):
    k_resid_gate(g, x, y, perm, topw, w_post, w_next, xn, 0, d, k, eps, gate, gate_b)
    _conv_rows(g[0], xn, w, out, state, lines, d, taps, line_bytes)


# ---- attention in a sliding window ----
def _window_pool(cache, dt, hk, page, d, dv):
    pool = cache.view(dt).view(-1, hk * page * (d + dv))
    return pool[:, : hk * page * d].unflatten(1, (hk, page, d)), pool[:, hk * page * d:].unflatten(1, (hk, page, dv))


def k_qk_prep(g, qkv, cache, positions, slots, cos, sin, qn, kn, hq, hk, d, dv, rot, halves, page, stride, max_pos, eps, err):
    n = g[0]
    rows, pos, sl = _rows(qkv, n, hq * d + hk * (d + dv), stride), positions[:n].long(), slots[:n].long()
    if ((pos < 0) | (pos >= max_pos)).any():
        err[0] = 300
    pos = torch.where((pos < 0) | (pos >= max_pos), 0, pos)
    c, s = (t.view(-1)[: max_pos * (rot // 2)].view(max_pos, rot // 2)[pos][:, None] for t in (cos, sin))

    def turned(x, w):
        x = _norm(x, w[:d], eps) if isinstance(w, T) else x
        a, b = (x[..., : rot // 2], x[..., rot // 2: rot]) if halves else (x[..., :rot:2], x[..., 1:rot:2])
        a, b = a * c - b * s, b * c + a * s
        return torch.cat([a, b, x[..., rot:]] if halves else [torch.stack([a, b], -1).flatten(-2), x[..., rot:]], -1)

    q = turned(_f(rows[:, : hq * d]).view(n, hq, d), qn)
    k = turned(_f(rows[:, hq * d:(hq + hk) * d]).view(n, hk, d), kn).to(qkv.dtype)
    v = rows[:, (hq + hk) * d:].reshape(n, hk, dv).clone()
    rows[:, : hq * d] = q.reshape(n, -1).to(qkv.dtype)
    ks, vs = _window_pool(cache, qkv.dtype, hk, page, d, dv)
    ok = sl >= 0
    ks[sl[ok] // page, :, sl[ok] % page] = k[ok]
    vs[sl[ok] // page, :, sl[ok] % page] = v[ok]


def k_qk_prep_whole(g, qkv, cache, positions, slots, cos, sin, qn, kn, hq, hk, d, dv, v_col, rot, halves, page, stride, max_pos, eps, err):
    n = g[0]
    rows, pos, sl = _rows(qkv, n, max((hq + hk) * d, v_col + hk * dv), stride), positions[:n].long(), slots[:n].long()
    if ((pos < 0) | (pos >= max_pos)).any():
        err[0] = 300
    pos = torch.where((pos < 0) | (pos >= max_pos), 0, pos)
    c, s = (t.view(-1)[: max_pos * (rot // 2)].view(max_pos, rot // 2)[pos][:, None] for t in (cos, sin))

    def turned(x, w, heads):
        x = _norm(_f(x), w[: heads * d], eps).view(n, heads, d)
        a, b = (x[..., : rot // 2], x[..., rot // 2: rot]) if halves else (x[..., :rot:2], x[..., 1:rot:2])
        a, b = a * c - b * s, b * c + a * s
        return torch.cat([a, b, x[..., rot:]] if halves else [torch.stack([a, b], -1).flatten(-2), x[..., rot:]], -1).to(qkv.dtype)

    q, k = turned(rows[:, : hq * d], qn, hq), turned(rows[:, hq * d:(hq + hk) * d], kn, hk)
    v = rows[:, v_col: v_col + hk * dv].reshape(n, hk, dv).clone()
    rows[:, : hq * d] = q.reshape(n, -1)
    ks, vs = _window_pool(cache, qkv.dtype, hk, page, d, dv)
    ok = sl >= 0
    ks[sl[ok] // page, :, sl[ok] % page] = k[ok]
    vs[sl[ok] // page, :, sl[ok] % page] = v[ok]


def _window_row(q, cache, out, pages, L, sink, hq, hk, d, dv, page, window, scale, cap, out_scale, gate=None):
    """One row at position L - 1: q [hq d] -> out [hq dv]. No cap (0), no sink (a score of 0) and no gate are forms too."""
    ks, vs = _window_pool(cache, q.dtype, hk, page, d, dv)
    ids = pages[: -(-L // page)].long()
    k, v = (_f(t[ids]).transpose(1, 2).reshape(-1, hk, t.shape[-1])[max(0, L - window):L].repeat_interleave(hq // hk, 1) for t in (ks, vs))
    s = torch.einsum("hd,lhd->hl", _f(q).view(hq, d), k) * scale
    s = cap * torch.tanh(s / cap) if cap > 0 else s
    sk = _f(sink[:hq]) if isinstance(sink, T) else torch.zeros(hq)
    p = torch.softmax(torch.cat([s, sk[:, None]], 1), 1)[:, :-1]
    o = (torch.einsum("hl,lhv->hv", p, v) * out_scale).reshape(-1)
    out.copy_(o * torch.sigmoid(_f(gate)) if gate is not None else o)


def _gate_row(gate, r, gs, cols):
    return gate[r * gs: r * gs + cols] if isinstance(gate, T) else None


def k_window_attn(g, q, cache, out, table, lens, row_seq, sink, gate, hq, hk, d, dv, qs, os_, gs, max_pages, page, window, scale, cap, out_scale, err):
    tb = table.view(-1, max_pages)
    for r in range(g[1]):
        if int(lens[r]) > 0:
            _window_row(q[r * qs: r * qs + hq * d], cache, out[r * os_: r * os_ + hq * dv], tb[int(row_seq[r]) if isinstance(row_seq, T) else r], int(lens[r]), sink,
                        hq, hk, d, dv, page, window, scale, cap, out_scale, _gate_row(gate, r, gs, hq * dv))


def _window_listed(q, cache, out, table, lens, cu, work, count, tokens, sink, hq, hk, d, qs, os_, max_pages, page, window, c1, c2, out_scale, gate=0, gs=0):
    """The rows of a work list's (sequence, block) pairs, `tokens` to a block; without a list, one row per sequence. c2 0: no cap,
    and c1 is the scale in base-2 units."""
    cap, tb = c2 / 1.4426950408889634, table.view(-1, max_pages)
    scale = c1 * cap / (2 * 1.4426950408889634) if cap else c1 / 1.4426950408889634
    pairs = work.view(-1, 2)[: int(count[0])].tolist()
    for s, b in pairs:
        r0, r1 = int(cu[s]), int(cu[s + 1])
        for t in range(b * tokens, min((b + 1) * tokens, r1 - r0)):
            r = r0 + t
            _window_row(q[r * qs: r * qs + hq * d], cache, out[r * os_: r * os_ + hq * d], tb[s], int(lens[s]) - (r1 - r0) + t + 1, sink, hq, hk, d, d, page, window,
                        scale, cap, out_scale, _gate_row(gate, r, gs, hq * d))


def _k_window(prefill, d):
    def run(g, kv, q, out, ws_o, ws_ml, table, lens, cu, work, count, hq, hk, qs, os_, max_pages, page, splits, pool_pages, err, sink, window, c1, c2, out_scale):
        if isinstance(work, T):
            _window_listed(q, kv, out, table, lens, cu, work, count, (64 if prefill else 16) // (hq // hk), sink, hq, hk, d, qs, os_, max_pages, page, window, c1, c2, out_scale)
        else:      # a split launch is followed by the merge; here it writes the finished rows and the merge is a no-op
            _window_listed(q, kv, out, table, lens, *_one_each(g[1], lens), 1, sink, hq, hk, d, qs, os_, max_pages, page, window, c1, c2, out_scale)
    return run


def _one_each(n, lens):
    """(row starts, list, count) of one row per sequence."""
    one = torch.arange(n + 1, dtype=torch.int32)
    live = [i for i in range(n) if int(lens[i]) > 0]
    return one, torch.stack([one[:-1], torch.zeros(n, dtype=torch.int32)], 1)[live].contiguous(), torch.tensor([len(live)])


WHOLE = 1 << 30


def _k_sink(prefill, d):
    def run(g, kv, q, out, ws_o, ws_ml, table, lens, cu, work, count, hq, hk, qs, os_, max_pages, page, splits, pool_pages, err, sink, gate, gs, scale_log2):
        if isinstance(work, T):
            rows = (cu, work, count, (64 if prefill else 16) // (hq // hk))
        else:
            rows = (*_one_each(g[1], lens), 1)
        _window_listed(q, kv, out, table, lens, *rows, sink, hq, hk, d, qs, os_, max_pages, page, WHOLE, scale_log2, 0.0, 1.0, gate, gs)
    return run


def _k_sink_ragged(d):
    def run(g, kv, q, out, table, lens, cu, wp, cp, wd, cd, hq, hk, qs, os_, max_pages, page, pool_pages, err, sink, gate, gs, scale_log2):
        for w, c, rows in ((wp, cp, 64), (wd, cd, 16)):
            _window_listed(q, kv, out, table, lens, cu, w, c, rows // (hq // hk), sink, hq, hk, d, qs, os_, max_pages, page, WHOLE, scale_log2, 0.0, 1.0, gate, gs)
    return run


def k_sink_fmha(g, kv, q, out, table, lens, cu, work, count, hq, hk, qs, os_, max_pages, page, pool_pages, err, sink, gate, gs, scale_log2):
    _window_listed(q, kv, out, table, lens, cu, work, count, 128 // (hq // hk), sink, hq, hk, 128, qs, os_, max_pages, page, WHOLE, scale_log2, 0.0, 1.0, gate, gs)


def _k_window_ragged(d):
    def run(g, kv, q, out, table, lens, cu, wp, cp, wd, cd, hq, hk, qs, os_, max_pages, page, pool_pages, err, sink, window, c1, c2, out_scale):
        for w, c, rows in ((wp, cp, 64), (wd, cd, 16)):
            _window_listed(q, kv, out, table, lens, cu, w, c, rows // (hq // hk), sink, hq, hk, d, qs, os_, max_pages, page, window, c1, c2, out_scale)
    return run


def k_window_fmha(g, kv, q, out, table, lens, cu, work, count, hq, hk, qs, os_, max_pages, page, pool_pages, err, sink, window, c1, c2, out_scale):
    _window_listed(q, kv, out, table, lens, cu, work, count, 128 // (hq // hk), sink, hq, hk, 128, qs, os_, max_pages, page, window, c1, c2, out_scale)


# ---- attention in a window beside pooled blocks ----
def _pooled_pool(pooled, dt, hk, slots, d, dv, stride):
    """(keys [pages, hk, slots, d], values) of the second cache, whose pages are `stride` bytes."""
    es, n = dt.itemsize, hk * slots * (d + dv)
    rows = torch.as_strided(pooled.view(dt), (pooled.numel() // stride, n), (stride // es, 1))
    return rows[:, : hk * slots * d].unflatten(1, (hk, slots, d)), rows[:, hk * slots * d:].unflatten(1, (hk, slots, dv))


def _pool_rows(n, cache, pooled, positions, slots, table, seq_of, hk, d, dv, page, pool, n_slots, stride, max_pages, dt):
    ks, vs = _window_pool(cache, dt, hk, page, d, dv)
    pk, pv = _pooled_pool(pooled, dt, hk, n_slots, d, dv, stride)
    tb = table.view(-1, max_pages)
    for t in range(n):
        pos, slot = int(positions[t]), int(slots[t])
        if slot < 0 or (pos + 1) % pool:
            continue
        b = pos // pool
        at = torch.arange(b * pool, pos + 1)
        pages, off = tb[seq_of(t)][at // page].long(), at % page
        place = b - pos // page * page // pool
        pk[slot // page, :, place] = _f(ks[pages, :, off]).mean(0).to(dt)
        pv[slot // page, :, place] = _f(vs[pages, :, off]).mean(0).to(dt)


def k_qk_prep_pool(g, qkv, cache, pooled, positions, slots, table, cos, sin, hq, hk, d, dv, rot, halves, page, stride, max_pos, pool, n_slots, pstride, max_pages, err):
    k_qk_prep(g, qkv, cache, positions, slots, cos, sin, 0, 0, hq, hk, d, dv, rot, halves, page, stride, max_pos, 0.0, err)
    _pool_rows(g[0], cache, pooled, positions, slots, table, lambda t: t, hk, d, dv, page, pool, n_slots, pstride, max_pages, qkv.dtype)


def _k_pool_blocks(dt):
    def run(g, cache, pooled, positions, slots, table, cu, seqs, rows, hk, d, dv, page, pool, n_slots, pstride, max_pages, err):
        seq_of = torch.repeat_interleave(torch.arange(seqs), (cu[1: seqs + 1] - cu[:seqs]).long()).tolist()
        _pool_rows(min(rows, len(seq_of)), cache, pooled, positions, slots, table, seq_of.__getitem__, hk, d, dv, page, pool, n_slots, pstride, max_pages, dt)
    return run


def _pooled_row(q, cache, pooled, out, pages, L, hq, hk, d, dv, page, window, pool, n_slots, pstride, scale):
    """One row at position L - 1: the window, and the blocks that end before it."""
    ks, vs = _window_pool(cache, q.dtype, hk, page, d, dv)
    pk, pv = _pooled_pool(pooled, q.dtype, hk, n_slots, d, dv, pstride)
    j = torch.arange(max(0, L - window), L)
    b = torch.arange(max(0, L - window) // pool)
    last = b * pool + pool - 1
    ids = lambda x: pages[x // page].long()
    place = b - last // page * page // pool
    k, v = (torch.cat([_f(pt[ids(last), :, place]), _f(t[ids(j), :, j % page])]).repeat_interleave(hq // hk, 1) for pt, t in ((pk, ks), (pv, vs)))
    s = torch.einsum("hd,lhd->hl", _f(q).view(hq, d), k) * scale
    out.copy_(torch.einsum("hl,lhv->hv", torch.softmax(s, 1), v).reshape(-1))


def k_pooled_attn(g, q, cache, pooled, out, table, lens, row_seq, hq, hk, d, dv, qs, os_, max_pages, page, window, pool, n_slots, pstride, scale, err):
    tb = table.view(-1, max_pages)
    for r in range(g[1]):
        if int(lens[r]) > 0:
            _pooled_row(q[r * qs: r * qs + hq * d], cache, pooled, out[r * os_: r * os_ + hq * dv], tb[int(row_seq[r]) if isinstance(row_seq, T) else r], int(lens[r]),
                        hq, hk, d, dv, page, window, pool, n_slots, pstride, scale)


def _pooled_listed(kv, pooled, q, out, table, lens, cu, work, count, tokens, hq, hk, d, qs, os_, max_pages, page, window, pool, n_slots, scale_log2):
    tb, pstride = table.view(-1, max_pages), 2 * hk * n_slots * d * q.element_size()
    for s, b in work.view(-1, 2)[: int(count[0])].tolist():
        r0, r1 = int(cu[s]), int(cu[s + 1])
        for t in range(b * tokens, min((b + 1) * tokens, r1 - r0)):
            r = r0 + t
            _pooled_row(q[r * qs: r * qs + hq * d], kv, pooled, out[r * os_: r * os_ + hq * d], tb[s], int(lens[s]) - (r1 - r0) + t + 1, hq, hk, d, d, page, window, pool,
                        n_slots, pstride, scale_log2 / 1.4426950408889634)


def _k_pooled(prefill, d):
    def run(g, kv, pooled, q, out, ws_o, ws_ml, table, lens, cu, work, count, hq, hk, qs, os_, max_pages, page, splits, pool_pages, err, window, pool, n_slots, sl2):
        # a split launch is followed by the merge; here it writes the finished rows and the merge is a no-op
        rows = (cu, work, count, (64 if prefill else 16) // (hq // hk)) if isinstance(work, T) else (*_one_each(g[1], lens), 1)
        _pooled_listed(kv, pooled, q, out, table, lens, *rows, hq, hk, d, qs, os_, max_pages, page, window, pool, n_slots, sl2)
    return run


def _k_pooled_ragged(d):
    def run(g, kv, pooled, q, out, table, lens, cu, wp, cp, wd, cd, hq, hk, qs, os_, max_pages, page, pool_pages, err, window, pool, n_slots, sl2):
        for w, c, rows in ((wp, cp, 64), (wd, cd, 16)):
            _pooled_listed(kv, pooled, q, out, table, lens, cu, w, c, rows // (hq // hk), hq, hk, d, qs, os_, max_pages, page, window, pool, n_slots, sl2)
    return run


def k_pooled_fmha(g, kv, pooled, q, out, table, lens, cu, work, count, hq, hk, qs, os_, max_pages, page, pool_pages, err, window, pool, n_slots, sl2):
    _pooled_listed(kv, pooled, q, out, table, lens, cu, work, count, 128 // (hq // hk), hq, hk, 128, qs, os_, max_pages, page, window, pool, n_slots, sl2)


# ---- latent attention ----
def k_latent_append(g, lat, cache, slots, w, rank, stride, eps):
    n = g[0]
    new = _norm(_f(_rows(lat, n, rank, stride)), w[:rank], eps).to(lat.dtype)
    sl = slots[:n].long()
    cache.view(lat.dtype).view(-1, rank)[sl[sl >= 0]] = new[sl >= 0]


def _attend(q, cache, out, table, lens, row_seq, rows, heads, rank, max_pages, page, scale):
    pool = cache.view(q.dtype).view(-1, page, rank)
    tb = table.view(-1, max_pages)
    for r in range(rows):
        n = int(lens[r])
        if n <= 0:
            continue
        pages = tb[int(row_seq[r]) if isinstance(row_seq, T) else r, : -(-n // page)].long()
        c = _f(pool[pages]).reshape(-1, rank)[:n]
        qq = _f(q[r * heads * rank:(r + 1) * heads * rank].view(heads, rank))
        out[r * heads * rank:(r + 1) * heads * rank] = (torch.softmax(qq @ c.t() * scale, -1) @ c).to(out.dtype).reshape(-1)


def k_latent_attn(g, q, cache, out, table, lens, row_seq, heads, rank, max_pages, page, scale, err):
    _attend(q, cache, out, table, lens, row_seq, g[1], heads, rank, max_pages, page, scale)


def k_latent_decode(g, kv, q, out, ws_o, ws_ml, table, lens, seqs, heads, qs, os_, max_pages, page, splits, pool_pages, scale_log2,
                    err, row_seq, rank):
    # a split launch is followed by the merge; here the first writes the finished rows and the merge is a no-op
    _attend(q, kv, out, table, lens, row_seq, g[1], heads, rank, max_pages, page, scale_log2 / 1.4426950408889634)


def _turn(x, pos, cos, sin, max_pos, rot, halves):
    """x [n, heads, rot], pairs (i, i + rot / 2) or neighbours, by the tables' rows `pos` [n]."""
    c, s = (t.view(-1)[: max_pos * (rot // 2)].view(max_pos, rot // 2)[pos][:, None] for t in (cos, sin))
    a, b = (x[..., : rot // 2], x[..., rot // 2:]) if halves else (x[..., ::2], x[..., 1::2])
    a, b = a * c - b * s, b * c + a * s
    return torch.cat([a, b], -1) if halves else torch.stack([a, b], -1).flatten(-2)


def k_latent_prep(g, rows, cache, q_low, positions, slots, cos, sin, w, wq, rank, rot, halves, q_rank, stride, qs, max_pos, eps, err):
    n = g[0]
    x, pos, sl = _f(_rows(rows, n, q_rank + rank + rot, stride)), positions[:n].long(), slots[:n].long()
    if ((pos < 0) | (pos >= max_pos)).any():
        err[0] = 300
    pos = torch.where((pos < 0) | (pos >= max_pos), 0, pos)
    _rows(q_low, n, q_rank, qs).copy_(_norm(x[:, :q_rank], wq[:q_rank], eps))
    key = _turn(x[:, None, q_rank + rank:], pos, cos, sin, max_pos, rot, halves)[:, 0]
    new = torch.cat([_norm(x[:, q_rank: q_rank + rank], w[:rank], eps), key], -1).to(rows.dtype)
    cache.view(rows.dtype).view(-1, rank + rot)[sl[sl >= 0]] = new[sl >= 0]


def _attend_rot(q, cache, out, table, lens, row_seq, n, heads, rank, rot, max_pages, page, scale, q_rot, cos, sin, sink, gate, rs, max_pos, halves, window, gs, err):
    pool = cache.view(q.dtype).view(-1, page, rank + rot)
    tb = table.view(-1, max_pages)
    for r in range(n):
        L = int(lens[r])
        if L <= 0:
            continue
        if L > max_pos:
            err[0] = 300
        c = _f(pool[tb[int(row_seq[r]) if isinstance(row_seq, T) else r, : -(-L // page)].long()]).reshape(-1, rank + rot)[max(0, L - window):L]
        turned = _turn(_f(q_rot[r * rs: r * rs + heads * rot].view(1, heads, rot)), torch.tensor([min(L, max_pos) - 1]), cos, sin, max_pos, rot, halves)[0]
        qq = torch.cat([_f(q[r * heads * rank:(r + 1) * heads * rank].view(heads, rank)), turned.to(q.dtype).float()], -1)
        s = qq @ c.t() * scale
        p = torch.softmax(torch.cat([s, _f(sink[:heads])[:, None]], 1), -1)[:, :-1] if isinstance(sink, T) else torch.softmax(s, -1)
        o = p @ c[:, :rank]
        o = o * torch.sigmoid(_f(gate[r * gs: r * gs + heads]))[:, None] if isinstance(gate, T) else o
        out[r * heads * rank:(r + 1) * heads * rank] = o.to(out.dtype).reshape(-1)


def k_latent_rot_attn(g, q, cache, out, table, lens, row_seq, heads, rank, max_pages, page, scale, err, q_rot, cos, sin, sink, gate, rs, rot, max_pos, halves, window, gs):
    _attend_rot(q, cache, out, table, lens, row_seq, g[1], heads, rank, rot, max_pages, page, scale, q_rot, cos, sin, sink, gate, rs, max_pos, halves, window, gs, err)


def k_latent_rot_decode(g, kv, q, out, ws_o, ws_ml, table, lens, seqs, heads, qs, os_, max_pages, page, splits, pool_pages, scale_log2, err, row_seq, rank,
                        q_rot, cos, sin, sink, gate, rs, rot, max_pos, halves, window, gs):
    # a split launch is followed by the merge; here the first writes the finished rows and the merge is a no-op
    _attend_rot(q, kv, out, table, lens, row_seq, g[1], heads, rank, rot, max_pages, page, scale_log2 / 1.4426950408889634, q_rot, cos, sin, sink, gate, rs, max_pos,
                halves, window, gs, err)


def k_route_table(g, ids, table, out, w, tokens, E, k, vocab, err):
    tok = ids[:tokens].long()
    ok = (tok >= 0) & (tok < vocab)
    rows = torch.where(ok[:, None], table[: vocab * k].view(vocab, k)[torch.where(ok, tok, 0)], -1)
    if ((rows < 0) | (rows >= E)).any():
        err[0] = 300
    out[: tokens * k] = rows.reshape(-1)
    w[: tokens * k] = 1.0 / k


def k_route_logits(g, logits, bias, ids, w, tokens, E, k, ld):
    z = _rows(logits, tokens, E, ld) + (_f(bias[:E]) if isinstance(bias, T) else 0.0)
    order = torch.argsort(z, dim=-1, descending=True, stable=True)[:, :k]
    ids[: tokens * k] = order.to(ids.dtype).reshape(-1)
    w[: tokens * k] = torch.softmax(torch.gather(z, 1, order), -1).reshape(-1)


def k_route_groups(g, logits, bias, ids, w, tokens, E, k, groups, keep, softmax, group_top, renorm, scale, ld):
    z = _rows(logits, tokens, E, ld)
    s = torch.softmax(z, -1) if softmax else torch.sigmoid(z)
    choice = s + _f(bias[:E]) if isinstance(bias, T) else s
    of = choice.view(tokens, groups, -1)
    best = torch.argsort(of.topk(min(group_top, E // groups), -1).values.sum(-1), dim=-1, descending=True, stable=True)[:, :keep]
    may = torch.zeros(tokens, groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(E // groups, 1)
    order = torch.argsort(choice.masked_fill(~may, -torch.inf), dim=-1, descending=True, stable=True)[:, :k]
    top = torch.gather(s, 1, order)
    ids[: tokens * k] = order.to(ids.dtype).reshape(-1)
    w[: tokens * k] = ((top / (top.sum(-1, keepdim=True) + 1e-20) if renorm else top) * scale).reshape(-1)


_DT = {"bf16": torch.bfloat16, "f32": torch.float32}
for _a in _DT:
    CPU_KERNELS.update({f"kern_hyper_embed_{_a}": k_hyper_embed, f"kern_row_norm_f32_{_a}": k_row_norm,
                        f"kern_rows_scatter_{_a}": k_rows_scatter, f"kern_gate_mul_{_a}": k_gate_mul,
                        f"kern_resid_embed_{_a}": k_resid_embed, f"kern_resid_mix_{_a}": k_resid_mix, f"kern_resid_embed_conv_{_a}": k_resid_embed_conv,
                        f"kern_resid_gate_{_a}": k_resid_gate, f"kern_resid_gate_conv_{_a}": k_resid_gate_conv, f"kern_conv_add_{_a}": k_conv_add,
                        f"kern_qk_prep_pool_{_a}": k_qk_prep_pool, f"kern_pool_blocks_{_a}": _k_pool_blocks(_DT[_a]),
                        f"kern_resid_scale_{_a}": k_resid_scale, f"kern_resid_scale_routed_{_a}": k_resid_scale, f"kern_qk_prep_whole_{_a}": k_qk_prep_whole, f"kern_latent_prep_{_a}": k_latent_prep,
                        f"kern_token_shift_{_a}": k_token_shift, f"kern_shift_state_{_a}": k_shift_state, f"kern_decay_{_a}": k_decay,
                        f"kern_lin_norm_gate_{_a}": k_lin_norm_gate, f"kern_qk_prep_{_a}": k_qk_prep,
                        f"kern_ssd_conv_{_a}": k_ssd_conv, f"kern_ssd_conv_state_{_a}": k_ssd_conv_state,
                        f"kern_ssd_gate_norm_{_a}": k_ssd_gate_norm, f"kern_latent_append_{_a}": k_latent_append})
    CPU_KERNELS.update({f"kern_hyper_{k}_{_a}_s{s}": f for s in range(5) for k, f in (("mix", k_hyper_mix), ("last", k_hyper_last))})
    CPU_KERNELS.update({f"kern_ssd_rule_{_a}_n{n}": k_ssd_rule for n in (32, 64, 128, 256, 512)})
    CPU_KERNELS.update({f"kern_{k}_{_a}{'_' + e if e else ''}": f(e) for k, f in (("linear", _k_linear), ("linear_grouped", _k_grouped))
                        for e in ("", "swiglu", "geglu", "clamped")})
    CPU_KERNELS.update({f"kern_lin_rule_{_a}_r{r}_v{v}": k_lin_rule for r in (4, 8, 16, 32) for v in (1, 2, 4)})
    CPU_KERNELS.update({f"kern_{k}_attn_{_a}_w{w}": f for k, f in (("window", k_window_attn), ("pooled", k_pooled_attn)) for w in (64, 128, 256, 512)})
    CPU_KERNELS.update({f"kern_latent_{n}_{_a}_w{w}": f for n, f in (("attn", k_latent_attn), ("rot_attn", k_latent_rot_attn)) for w in (64, 128, 256, 512, 1024)})
CPU_KERNELS.update({"kern_linear_bf16_f32": _k_linear(""), "kern_transpose_heads_bf16": k_transpose_heads, "kern_copy_cols_bf16": k_copy_cols,
                    "kern_moe_route_logits": k_route_logits, "kern_moe_route_groups": k_route_groups, "kern_attn_window_fmha_d128": k_window_fmha,
                    "kern_attn_sink_fmha_d128": k_sink_fmha, "kern_attn_pooled_fmha_d128": k_pooled_fmha, "kern_moe_route_table": k_route_table,
                    "kern_attn_window_merge": lambda *a: None, "kern_attn_gated_merge": lambda *a: None})
CPU_KERNELS.update({f"kern_moe_gemm_bf16_{e}_n{n}": _k_moe_gemm(e) for e in ("geglu", "clamped") for n in (64, 128)})
CPU_KERNELS.update({f"kern_lin_{k}_n{n}": f for k, f in (("prep", k_lin_prep), ("chunk", k_lin_chunk)) for n in (32, 64, 128, 256)})
CPU_KERNELS.update({f"kern_attn_window_{k}_d{d}": _k_window(k == "prefill", d) for k in ("decode", "prefill") for d in (64, 128, 256)})
CPU_KERNELS.update({f"kern_attn_window_ragged_d{d}": _k_window_ragged(d) for d in (64, 128)})
CPU_KERNELS.update({f"kern_attn_sink_{k}_d{d}": _k_sink(k == "prefill", d) for k in ("decode", "prefill") for d in (64, 128, 256)})
CPU_KERNELS.update({f"kern_attn_sink_ragged_d{d}": _k_sink_ragged(d) for d in (64, 128)})
CPU_KERNELS.update({f"kern_attn_pooled_{k}_d{d}": _k_pooled(k == "prefill", d) for k in ("decode", "prefill") for d in (64, 128, 256)})
CPU_KERNELS.update({f"kern_attn_pooled_ragged_d{d}": _k_pooled_ragged(d) for d in (64, 128)})
CPU_KERNELS.update({f"kern_gemm_bf16_heads_n{n}": k_gemm_heads for n in (64, 128, 256)})
CPU_KERNELS.update({f"kern_ssd_chunk_n{n}": k_ssd_chunk for n in (32, 64, 128, 256)})
CPU_KERNELS.update({f"kern_latent_decode_bf16_b{b}": k_latent_decode for b in range(1, 9)})
CPU_KERNELS.update({f"kern_latent_rot_decode_bf16_q{b + more}_b{b}": k_latent_rot_decode for b in range(1, 9) for more in (0, 1)})

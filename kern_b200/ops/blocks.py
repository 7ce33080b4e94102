"""CPU statements of the kernels in hyper.cu, linear.cu, ssd.cu, latent.cu (and the latent forms in mla_decode.cu / moe.cu):
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


# ---- matrix products ----
def _swiglu(v):
    half = v.shape[1] // 2
    return F.silu(v[:, :half]) * v[:, half:]


def _k_linear(swiglu):
    def run(g, a, w, c, m, n, k, lda, ldc, wsn, wsk, az, wz, cz, err):
        if m > g[1] * 64:
            err[0] = 300
        for z in range(g[2]):
            A = _f(_rows(a[z * az:], m, k, lda))
            W = _f(torch.as_strided(w[z * wz:], ((2 if swiglu else 1) * n, k), (wsn, wsk)))
            v = A @ W.t()
            _rows(c[z * cz:], m, n, ldc).copy_(_swiglu(v) if swiglu else v)
    return run


def k_gemm_heads(g, a, w, c, m, n, k, ldc, heads, err):
    lda = a._row_stride
    for h in range(heads):
        W = _f(w[h * n * k:(h + 1) * n * k].view(n, k))
        _rows(c[h * n:], m, n, ldc).copy_(_f(_rows(a[h * k:], m, k, lda)) @ W.t())


def _k_grouped(swiglu):
    def run(g, a, w, c, tiles, count, rows, n, k, wz, err):
        for e, r0, nr, _ in tiles.view(-1, 4)[: int(count[0])].tolist():
            W = _f(w[e * wz: e * wz + (2 if swiglu else 1) * n * k].view(-1, k))
            v = _f(a[r0 * k:(r0 + nr) * k].view(nr, k)) @ W.t()
            c[r0 * n:(r0 + nr) * n] = (_swiglu(v) if swiglu else v).to(c.dtype).reshape(-1)
    return run


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


def k_route_logits(g, logits, bias, ids, w, tokens, E, k, ld):
    z = _rows(logits, tokens, E, ld) + (_f(bias[:E]) if isinstance(bias, T) else 0.0)
    order = torch.argsort(z, dim=-1, descending=True, stable=True)[:, :k]
    ids[: tokens * k] = order.to(ids.dtype).reshape(-1)
    w[: tokens * k] = torch.softmax(torch.gather(z, 1, order), -1).reshape(-1)


for _a in ("bf16", "f32"):
    CPU_KERNELS.update({f"kern_hyper_embed_{_a}": k_hyper_embed, f"kern_row_norm_f32_{_a}": k_row_norm,
                        f"kern_rows_scatter_{_a}": k_rows_scatter, f"kern_gate_mul_{_a}": k_gate_mul,
                        f"kern_linear_{_a}": _k_linear(False), f"kern_linear_{_a}_swiglu": _k_linear(True),
                        f"kern_linear_grouped_{_a}": _k_grouped(False), f"kern_linear_grouped_{_a}_swiglu": _k_grouped(True),
                        f"kern_ssd_conv_{_a}": k_ssd_conv, f"kern_ssd_conv_state_{_a}": k_ssd_conv_state,
                        f"kern_ssd_gate_norm_{_a}": k_ssd_gate_norm, f"kern_latent_append_{_a}": k_latent_append})
    CPU_KERNELS.update({f"kern_hyper_{k}_{_a}_s{s}": f for s in range(5) for k, f in (("mix", k_hyper_mix), ("last", k_hyper_last))})
    CPU_KERNELS.update({f"kern_ssd_rule_{_a}_n{n}": k_ssd_rule for n in (32, 64, 128, 256, 512)})
    CPU_KERNELS.update({f"kern_latent_attn_{_a}_w{w}": k_latent_attn for w in (64, 128, 256, 512, 1024)})
CPU_KERNELS.update({"kern_linear_bf16_f32": _k_linear(False), "kern_transpose_heads_bf16": k_transpose_heads,
                    "kern_moe_route_logits": k_route_logits})
CPU_KERNELS.update({f"kern_gemm_bf16_heads_n{n}": k_gemm_heads for n in (64, 128, 256)})
CPU_KERNELS.update({f"kern_ssd_chunk_n{n}": k_ssd_chunk for n in (32, 64, 128, 256)})
CPU_KERNELS.update({f"kern_latent_decode_bf16_b{b}": k_latent_decode for b in range(1, 9)})

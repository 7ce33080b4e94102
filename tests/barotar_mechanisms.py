"""Each mechanism alone against its plain statement: bodies shared by the CPU and the GPU tests."""
import torch

from kern_b200.models import blocks as K
from kern_b200.models import common as C
from tests.gafapel_cases import run_op
from tests.gafapel_mechanisms import DT, bf, close, rnd
from tests.oracles import barotar as O

i32 = lambda *s: torch.zeros(*s, dtype=torch.int32)
ints = lambda v: torch.tensor(v, dtype=torch.int32)


def resid_embed(gpu, act, width):
    n, vocab = 7, 31
    ids, table, w = torch.arange(n) * 5 % vocab, bf(rnd(vocab, width)), bf(1 + rnd(width, seed=1, scale=.1))
    out = run_op(K.resid_embed_op(width, vocab, 1e-5, act), [ids, table, w, torch.zeros(n, width), torch.zeros(n, width, dtype=DT[act]), i32(1)], gpu, {"tokens": n})
    x = table.double()[ids]
    assert torch.equal(out[3].double(), x) and int(out[5]) == 0
    close(out[4], O.rms(x, 1e-5) * w.double(), act)


def resid(gpu, act, width, routed):
    n, k = 6, max(1, routed)
    x, post, nxt = rnd(n, width), bf(1 + rnd(width, seed=1, scale=.3)), bf(1 + rnd(width, seed=2, scale=.3))
    y = rnd(n * k, width, seed=3, scale=4).to(DT[act])
    perm, tw = torch.randperm(n * k, generator=torch.Generator().manual_seed(4)).int(), rnd(n, k, seed=5).sigmoid()
    extra = [perm, tw] if routed else []
    yv = (y[perm.long()].double().view(n, k, width) * tw.double()[..., None]).sum(1) if routed else y.double()
    new = x.double() + O.rms(yv, 1e-4) * post.double()
    out = run_op(K.resid_mix_op(width, 1e-4, act, routed), [x, y, post, nxt, torch.zeros(n, width, dtype=DT[act]), *extra], gpu, {"tokens": n})
    close(out[0], new, "f32")
    close(out[4], O.rms(new, 1e-4) * nxt.double(), act)
    out = run_op(K.resid_mix_op(width, 1e-4, act, routed, last=True), [x, y, post, torch.zeros(n, width), *extra], gpu, {"tokens": n})
    close(out[3], new, "f32")


def glu(gpu, act, m, n, k, kind):
    a, w, limit = rnd(m, k).to(DT[act]), bf(rnd(2 * n, k, seed=1, scale=3 * k ** -0.5)), 1.7
    v = a.double() @ w.double().t()
    g, u = v[:, :n], v[:, n:]
    if kind == "geglu":
        want = O.gelu(g) * u
    else:
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        want = g * O.sigmoid(1.702 * g) * (u + 1)
    op = K.linear_op(2 * n, k, act=act, epilogue=kind, rows_max=max(m, 300), limit=limit)
    out = run_op(op, [a, w, torch.zeros(m, n, dtype=DT[act]), m, i32(1)], gpu, {"tokens": m})
    close(out[2], want, act)
    assert int(out[4]) == 0


def route(gpu, experts, top, groups, keep):
    z = rnd(40, experts, scale=2)
    z[3] = -rnd(experts, seed=3).abs() * 40          # scores that nearly vanish
    out = run_op(K.route_groups_op(experts, top, groups, keep), [z, i32(40, top), torch.zeros(40, top), 40], gpu, {"tokens": 40})
    shut = 0
    for t, chosen in enumerate(O.route(z.double(), top, groups, keep)):
        assert [e for e, _ in chosen] == out[1][t].tolist(), t
        close(out[2][t], torch.stack([v for _, v in chosen]), "f32")
        shut += [e for e, _ in chosen] != z[t].double().argsort(descending=True)[:top].tolist()
    assert (shut > 0) == (keep < groups < experts)   # the groups decide, where there are any to leave out (groups of one: top <= keep)


def routed_experts(gpu, act, width, ff, experts, top, groups, keep, n):
    x = rnd(n, width).to(DT[act])
    wr, limit = bf(rnd(experts, width, seed=1, scale=2 * width ** -0.5)), 1.1
    w = {"router": wr}
    for e in range(experts):
        for t, (r, c) in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            w[f"e{e}.{t}"] = bf(rnd(r, c, seed=10 + e * 3 + len(t), scale=(2 if t != "down" else 1) * c ** -0.5))
    ops, tokens = K.routed_ops(width, ff, experts, top, 300, act, "clamped", limit), {"tokens": n}
    r = run_op(K.route_groups_op(experts, top, groups, keep), [x.float() @ wr.float().t(), i32(n, top), torch.zeros(n, top), n], gpu, tokens)
    tiles = 300 * top // K.routed_tile_rows(act, width, ff) + experts
    p = run_op(ops["moe_plan"], [r[1], i32(n, top), i32(experts + 1), i32(tiles, 4), i32(1), i32(1), n * top, i32(1)], gpu, tokens)
    assert sorted(p[1].view(-1).tolist()) == list(range(n * top)) and int(p[7]) == 0
    g = run_op(ops["moe_gather"], [x, p[1], torch.zeros(300 * top, width, dtype=DT[act]), n * top], gpu, tokens)
    w1 = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)])
    w2 = torch.stack([w[f"e{e}.down"] for e in range(experts)])
    a = run_op(ops["moe_fc1"], [g[2], w1, torch.zeros(300 * top, ff, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)
    y = run_op(ops["moe_fc2"], [a[2], w2, torch.zeros(300 * top, width, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)
    got = (y[2][p[1].long()].float() * r[2][..., None]).sum(1)
    m = {"router": {"top": top, "groups": {"count": groups, "keep": keep}}, "expert": {"limit": limit}}
    close(got, O.experts({k: v.double() for k, v in w.items()}, "", m, x.double()), act)


def copy_cols(gpu):
    a, b = bf(rnd(9, 13)), bf(rnd(9, 21, seed=1))
    dst = torch.zeros(9 * 34, dtype=torch.bfloat16)
    dst = run_op(K.copy_cols_op(9, 13, 34), [a, dst], gpu)[1]
    view = torch.cat([dst[13:], torch.zeros(13, dtype=torch.bfloat16)])      # the columns from 13 on, as an argument with an offset sees them
    out = run_op(K.copy_cols_op(9, 21, 34), [b, view], gpu)[1]
    assert torch.equal(dst.view(9, 34)[:, :13], a) and torch.equal(out.view(9, 34)[:, :21], b)


def shift(gpu, act, width, targets, chunks, ragged):
    """Three sequences in chunks against whole ones; the lines end with each one's last row, other lines stay as they were."""
    lens, dt = [sum(c) for c in chunks], DT[act]
    h, mu = [rnd(n, width, seed=i).to(dt) for i, n in enumerate(lens)], bf(rnd(targets, width, seed=9).sigmoid())
    want = [torch.stack([O.shifted(x.double(), torch.zeros(width, dtype=torch.float64), m.double()) for m in mu], 1) for x in h]
    line = (width * 4 + 255) // 256 * 256 + 256
    state, lines, at = torch.zeros(5 * line, dtype=torch.uint8), ints([3, 1, 4]), [0, 0, 0]
    op = K.token_shift_op(width, targets, line, ragged, act)
    for step in zip(*chunks):
        rows = torch.cat([h[i][at[i]:at[i] + n] for i, n in enumerate(step)])
        cu = ints([0, *torch.tensor(step).cumsum(0).tolist()])
        out = run_op(op, [rows, mu, torch.zeros(len(rows), targets, width, dtype=dt), state, lines, *([cu] if ragged else []), 3], gpu,
                     {"tokens": len(rows), "seqs": 3})
        state = out[3]
        close(out[2], torch.cat([want[i][at[i]:at[i] + n] for i, n in enumerate(step)]), act)
        at = [a + n for a, n in zip(at, step)]
    for i, ln in enumerate(lines.tolist()):
        assert torch.equal(state[ln * line: ln * line + width * 4].view(torch.float32).double(), h[i][-1].double())
    assert int(state[:line].sum()) == 0 and int(state[2 * line:3 * line].sum()) == 0


def decay(gpu, act, rows, n, rank, kind):
    lda = rank + 3
    a, w, b = rnd(rows, lda, scale=2).to(DT[act]), bf(rnd(n, rank, seed=1, scale=2 * rank ** -0.5)), bf(rnd(n, seed=2, scale=3))
    b[0], b[n - 1] = 60, -60                          # saturated on either side
    out = run_op(K.decay_op(n, rank, lda, kind, 7.0, act), [a, w, b, torch.zeros(rows, n), rows], gpu, {"tokens": rows})
    x = a[:, :rank].double()
    if kind == "root":
        want = O.gla_decay(x @ w.double().t() + b.double(), 7.0)
    else:
        want = O.rwkv_decay(torch.tanh(x) @ w.double().t() + b.double())
    close(out[3], want, "f32")


def rule(gpu, act, H, dk, dv, chunks, ragged, bonus):
    """Two sequences in chunks against whole ones, alone on their lines. Decays reach from exactly 0 and nearly 1 to everything
    between, channel by channel and token by token."""
    lens, dt = [sum(c) for c in chunks], DT[act]
    fused, stride = not ragged and K.lin_fused(dv), 2 * H * dk + 2 * H * dv + 8
    proj = [rnd(n, stride, seed=i).to(dt) for i, n in enumerate(lens)]
    alpha = [torch.exp(-torch.exp(rnd(n, H * dk, seed=10 + i, scale=2.5) - 2)) for i, n in enumerate(lens)]
    for a in alpha:
        a[::7, ::3], a[1::5, 1::4] = 0, 1
    u, norm = bf(rnd(H, dk, seed=20)), bf(1 + rnd(*((H, dv) if bonus else (dv,)), seed=21, scale=.2))
    scale, out_scale, eps = 0.4, 0.7, 1e-5
    cols = lambda x, c, w: x[:, c:c + H * w].reshape(-1, H, w).double()
    want = []
    for i in range(2):
        q, k, v = cols(proj[i], 0, dk) * scale, cols(proj[i], H * dk, dk), cols(proj[i], 2 * H * dk, dv)
        a, S = alpha[i].double().view(-1, H, dk), torch.zeros(H, dk, dv, dtype=torch.float64)
        want.append(O.rwkv_rule(q, k, v, a, u.double(), S) if bonus else O.gla_rule(q, k, v, a, S))
    gated = lambda o, x: (O.rms(o, eps) * norm.double() * out_scale * O.silu(cols(x, 2 * H * dk + H * dv, dv))).reshape(-1, H * dv)
    s_off, os_ = 256, H * dv + 5
    line = 256 + (H * dk * dv * 4 + 255) // 256 * 256
    state, lines, at = torch.zeros(4 * line, dtype=torch.uint8), ints([3, 1]), [0, 0]
    op = K.lin_rule_op(H, dk, dv, stride, line, s_off, ragged, act, bonus=bonus, q_scale=scale, fused=fused, norm_shared=not bonus, out_stride=os_, out_scale=out_scale, eps=eps,
                       rows_max=140, seqs_max=2)
    ng = K.lin_norm_gate_op(H, dv, stride, not bonus, os_, out_scale, eps, act)
    for step in zip(*chunks):
        n = sum(step)
        x = torch.cat([proj[i][at[i]:at[i] + k] for i, k in enumerate(step)])
        al = torch.cat([alpha[i][at[i]:at[i] + k] for i, k in enumerate(step)])
        col = lambda c: torch.cat([x.view(-1)[c:], torch.zeros(c, dtype=dt)])
        q, k_, v, gate = x, col(H * dk), col(2 * H * dk), col(2 * H * dk + H * dv)
        out_t = torch.zeros(n, os_, dtype=dt) if fused else torch.zeros(n, H * dv)
        cu = [ints([0, step[0], n])] if ragged else []
        tokens = {"tokens": n, "seqs": 2}
        out = run_op(op, [q, k_, v, al, *([u] if bonus else []), out_t, state, lines, *cu, *([gate, norm] if fused else []), 2], gpu, tokens)
        got, state = out[4 + bonus], out[5 + bonus]
        o = torch.cat([want[i][0][at[i]:at[i] + k] for i, k in enumerate(step)])
        if not fused:
            close(got, o.reshape(n, -1), "f32", 5)
            got = run_op(ng, [got, gate, norm, torch.zeros(n, os_, dtype=dt)], gpu, tokens)[3]
        close(got[:, :H * dv], gated(o, x), act)
        assert not got[:, H * dv:].any()
        at = [a + k for a, k in zip(at, step)]
    for i, ln in enumerate(lines.tolist()):
        close(state[ln * line + s_off: ln * line + s_off + H * dk * dv * 4].view(torch.float32).view(H, dk, dv), want[i][1], "f32", 5)
    assert int(state[:line].sum()) == 0 and int(state[2 * line:3 * line].sum()) == 0


def prep(gpu, act, hq, hk, d, dv, rot, halves):
    n, page, dt, stride, pos_max = 6, 16, DT[act], hq * d + hk * (d + dv) + 8, 400
    qkv, pos, slots = rnd(n, stride, scale=3).to(dt), torch.tensor([0, 1, 399, 17, 64, 5]), torch.tensor([17, 0, -1, 47, 5, 16])
    qn, kn = bf(1 + rnd(d, seed=1, scale=.4)), bf(1 + rnd(d, seed=2, scale=.4))
    cache = torch.zeros(4 * hk * page * (d + dv) * dt.itemsize, dtype=torch.uint8)
    base = 300.0
    tabs = run_op(C.rope_table_op(pos_max, rot, base), [torch.zeros(pos_max, rot // 2), torch.zeros(pos_max, rot // 2)], gpu)
    out = run_op(K.qk_prep_op(hq, hk, d, dv, rot, page, stride, pos_max, 1e-4, act, halves), [qkv, cache, pos, slots, tabs[0], tabs[1], qn, kn, i32(1)], gpu, {"tokens": n})
    order = torch.arange(d)
    if halves:      # the same rotation over columns in another order
        order[:rot] = torch.arange(rot).view(2, -1).t().reshape(-1)
    turn = lambda x, w: O.rotate((O.rms(x.double(), 1e-4) * w.double())[..., order], pos, rot, base)[..., torch.argsort(order)]
    close(out[0][:, : hq * d], turn(qkv[:, : hq * d].reshape(n, hq, d), qn).reshape(n, -1), act)
    assert torch.equal(out[0][:, hq * d:], qkv[:, hq * d:]) and int(out[8]) == 0
    pool = out[1].view(dt).view(4, hk * page * (d + dv))
    ks, vs = pool[:, : hk * page * d].view(4, hk, page, d), pool[:, hk * page * d:].view(4, hk, page, dv)
    ok = slots >= 0
    close(ks[slots[ok] // page, :, slots[ok] % page], turn(qkv[:, hq * d:(hq + hk) * d].reshape(n, hk, d), kn)[ok], act)
    assert torch.equal(vs[slots[ok] // page, :, slots[ok] % page], qkv[:, (hq + hk) * d:(hq + hk) * d + hk * dv].reshape(n, hk, dv)[ok])
    rest = [i for i in range(64) if i not in slots.tolist()]
    assert not ks.transpose(1, 2).reshape(64, -1)[rest].any() and not vs.transpose(1, 2).reshape(64, -1)[rest].any()


def attention(gpu, act, hq, hk, d, dv, window, page, seqs, ragged):
    """`seqs`: (context, new rows) of every sequence, over scattered pages. Every row and head has a key that stands far out, its
    place by turns: the oldest the window keeps, the one just outside it (which must not be seen), the row's own, the first of
    all, the last of the page before and the one after the row (another row's, unseen too)."""
    width, dt, scale, cap, out_scale = 40, DT[act], 0.35, 8.0, 1.3
    rows = [(s, L - R + i) for s, (L, R) in enumerate(seqs) for i in range(R)]
    n, qs, os_ = len(rows), hq * d + 16, hq * dv + 8
    pages = sum(-(-L // page) for L, _ in seqs) + 3
    order, at = torch.randperm(pages, generator=torch.Generator().manual_seed(3)).tolist(), 0
    ks, vs = rnd(pages, hk, page, d, seed=4, scale=.5).to(dt), rnd(pages, hk, page, dv, seed=5).to(dt)
    table = torch.zeros(len(seqs), width, dtype=torch.int32)
    for s, (L, _) in enumerate(seqs):
        for i in range(-(-L // page)):
            table[s, i] = order[at]
            at += 1
    flat = lambda t, s: torch.cat([t[table[s, i]] for i in range(-(-seqs[s][0] // page))], 1)[:, :seqs[s][0]].transpose(0, 1)      # [L, hk, *]
    sink = bf(6.5 + rnd(hq, seed=6, scale=2))
    q = rnd(n, hq, d, seed=7, scale=.3)
    kf = [flat(ks, s).float() for s in range(len(seqs))]
    vf = [flat(vs, s).double() for s in range(len(seqs))]
    for r, (s, p) in enumerate(rows):
        for h in range(hq):
            j = [p - window + 1, p - window, p, 0, p // page * page - 1, p + 1][(r + h) % 6]
            j = min(max(j, 0), seqs[s][0] - 1)
            c = kf[s][j, h // (hq // hk)]
            q[r, h] += 14 * c / c.pow(2).sum() ** 0.5
    q = q.to(dt)
    buf = torch.zeros(n, qs, dtype=dt)
    buf[:, : hq * d] = q.view(n, -1)
    cache = torch.cat([ks.reshape(pages, -1), vs.reshape(pages, -1)], 1).contiguous().view(torch.uint8).view(-1)
    tiled = K.window_tiles(hq, hk, d, dv, page, act)
    vars_ = {"tokens": n, "seqs": len(seqs)}
    lens, extra = ints([L for L, _ in seqs]), []
    if ragged and tiled:
        cu = ints([0, *torch.tensor([R for _, R in seqs]).cumsum(0).tolist()])
        items = n // (64 // (hq // hk)) + len(seqs) + 1
        plan = run_op(C.attn_plan_op(hq, hk, len(seqs), d), [cu, i32(items, 2), i32(1), len(seqs), items, i32(len(seqs), 2), i32(1)], gpu, vars_)
        extra = [cu, plan[1], plan[2], plan[5], plan[6]]
    elif ragged:
        lens, extra = ints([p + 1 for _, p in rows]), [ints([s for s, _ in rows])]
    op = K.window_attn_op(hq, hk, d, dv, window, scale, cap, page, width, qs, os_, out_scale, ragged, act, seqs_max=len(seqs))
    out = run_op(op, [buf, cache, torch.zeros(n, os_, dtype=dt), table, lens, sink, i32(1), *extra], gpu, vars_)
    want = [O.window_attend(q[r:r + 1].double(), kf[s][:p + 1].double(), vf[s][:p + 1], scale, cap, window, sink.double())[0].reshape(-1) * out_scale
            for r, (s, p) in enumerate(rows)]
    close(out[2][:, : hq * dv], torch.stack(want), act)
    assert not out[2][:, hq * dv:].any() and int(out[6]) == 0
    # the oracle with the window one token longer or shorter, or without the sink, is far away: the limits see each
    some = [r for r, (_, p) in enumerate(rows) if p >= window][:6]
    for size, sk in ((window + 1, sink), (window - 1, sink), (window, sink - 1e4)):
        off = [0.0]
        for r in some if size else ():
            s, p = rows[r]
            other = O.window_attend(q[r:r + 1].double(), kf[s][:p + 1].double(), vf[s][:p + 1], scale, cap, size, sk.double())[0].reshape(-1) * out_scale
            off.append(float((other - want[r]).abs().max() / want[r].abs().max()))
        assert max(off) > 0.04 or len(off) * hq < 7, (size, off)

"""Each mechanism alone against its plain statement: bodies shared by the CPU and the GPU tests."""
import torch

from kern_b200.models import blocks as K
from kern_b200.models import common as C
from tests.gafapel_cases import run_op
from tests.gafapel_mechanisms import DT, bf, close, rnd
from tests.oracles import diderax as O

i32 = lambda *s: torch.zeros(*s, dtype=torch.int32)
ints = lambda v: torch.tensor(v, dtype=torch.int32)


def rope_table(gpu, dims, base, factor):
    """The tables turn a row of ones and zeros as the rotation does, also at far positions."""
    n, half = 4000, dims // 2
    out = run_op(C.rope_table_op(n, dims, base, factor), [torch.zeros(n, half), torch.zeros(n, half)], gpu)
    x = torch.cat([torch.ones(n, 1, half), torch.zeros(n, 1, half)], -1).double()
    want = O.rotate(x, torch.arange(n), dims, base, factor)[:, 0]
    close(torch.cat([out[0], out[1]], -1), want, "f32", 0.1)
    if factor != 1:
        assert float((O.rotate(x, torch.arange(n), dims, base)[:, 0] - want).abs().max()) > 0.1


def resid_scale(gpu, act, width, kind):
    """kind: plain, bias, routed (every choice has a row), identity (some do not; one token's are all without), shared."""
    n, k = 6, 3 if kind in ("routed", "identity", "shared") else 1
    x, s, nxt = rnd(n, width), bf(1 + rnd(width, seed=1, scale=.3)), bf(1 + rnd(width, seed=2, scale=.3))
    y, h = rnd(n * k, width, seed=3, scale=2).to(DT[act]), rnd(n, width, seed=9).to(DT[act])
    perm, tw = torch.randperm(n * k, generator=torch.Generator().manual_seed(4)).int().view(n, k), rnd(n, k, seed=5).sigmoid()
    b, sh, gate = bf(rnd(width, seed=6)), rnd(n, width, seed=7).to(DT[act]), rnd(n, 11, seed=8, scale=3)
    if kind in ("identity", "shared"):
        perm[0, 1] = perm[2, 0] = perm[2, 2] = -1
        perm[4] = -1
    routed = k if k > 1 else 0
    if routed:
        rows = torch.where((perm < 0)[..., None], h.double()[:, None], y.double()[perm.long().clamp_min(0)])
        v = (rows * tw.double()[..., None]).sum(1)
    else:
        v = y.double()
    extra, kw = [], {}
    if kind == "bias":
        extra, kw, v = [b], {"bias": True}, v + b.double()
    if routed:
        extra, kw = [perm, tw], {"routed": routed}
    if kind == "shared":
        extra, kw = [*extra, sh, gate], {**kw, "shared_gate": 11}
        v = v + sh.double() * O.sigmoid(gate[:, :1].double())
    new = x.double() + s.double() * v
    out = run_op(K.resid_scale_op(width, 1e-4, act, **kw), [x, y, s, nxt, h, *extra], gpu, {"tokens": n})
    close(out[0], new, "f32")
    close(out[4], O.rms(new, 1e-4) * nxt.double(), act)
    out = run_op(K.resid_scale_op(width, 1e-4, act, last=True, **kw), [x, y, s, torch.zeros(n, width), *extra, *([h] if routed else [])], gpu, {"tokens": n})
    close(out[3], new, "f32")


def glu_bias(gpu, act, m, n, k):
    a, w, b = rnd(m, k).to(DT[act]), bf(rnd(2 * n, k, seed=1, scale=3 * k ** -0.5)), bf(rnd(2 * n, seed=2, scale=2))
    v = a.double() @ w.double().t() + b.double()
    op = K.linear_op(2 * n, k, act=act, epilogue="swiglu", rows_max=max(m, 300), bias=True)
    out = run_op(op, [a, w, torch.zeros(m, n, dtype=DT[act]), m, i32(1), b], gpu, {"tokens": m})
    close(out[2], O.silu(v[:, :n]) * v[:, n:], act)
    assert int(out[4]) == 0


def route(gpu, outputs, top, groups, keep, scale):
    """Corrections of the scores' own size, some far below zero: the choice goes by them, the weights do not."""
    ld = outputs + 3
    z, c = rnd(60, ld, scale=2), bf(rnd(outputs, seed=1, scale=1.5 / outputs))
    c[::3] -= 0.7                                    # choices below zero
    z[3] = -rnd(ld, seed=3).abs() * 40               # all but one vanish
    op = K.route_groups_op(outputs, top, groups, keep, True, softmax=True, correction=True, group_top=1, scale=scale, ld=ld)
    out = run_op(op, [z, c, i32(60, top), torch.zeros(60, top), 60], gpu, {"tokens": 60})
    moved = shut = 0
    for t, chosen in enumerate(O.route(z[:, :outputs].double(), c.double(), top, groups, keep, scale)):
        ids = [e for e, _ in chosen]
        assert ids == out[2][t].tolist(), t
        close(out[3][t], torch.stack([v for _, v in chosen]), "f32")
        s = torch.softmax(z[t, :outputs].double(), -1)
        moved += sorted(ids) != sorted(s.argsort(descending=True)[:top].tolist())
        shut += sorted(ids) != sorted((s + c.double()).argsort(descending=True)[:top].tolist())
    assert (moved > 0) == (top < outputs) and (shut > 0 or keep == groups or top == 1 or groups == outputs)


def routed_experts(gpu, act, width, ff, experts, identity, top, groups, keep, n):
    """Router to weighted rows: some choices have no row and hand back the input."""
    outputs, x = experts + identity, rnd(n, width).to(DT[act])
    w = {"router": bf(rnd(outputs, width, seed=1, scale=2 * width ** -0.5)), "correction": bf(rnd(outputs, seed=2, scale=.5 / outputs)),
         "shared.sg": bf(rnd(1, width, seed=3, scale=2 * width ** -0.5))}
    for j, e in enumerate([*(f"e{e}" for e in range(experts)), "shared"]):
        for t, (r, c) in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            w[f"{e}.{t}"] = bf(rnd(r, c, seed=10 + j * 3 + len(t), scale=(2 if t != "down" else 1) * c ** -0.5))
    ops, tokens = K.routed_ops(width, ff, experts, top, 300, act), {"tokens": n}
    logits = torch.cat([x.float() @ w["router"].float().t(), x.float() @ w["shared.sg"].float().t()], 1)
    op = K.route_groups_op(outputs, top, groups, keep, True, softmax=True, correction=True, group_top=1, scale=1.3, ld=outputs + 1)
    r = run_op(op, [logits, w["correction"], i32(n, top), torch.zeros(n, top), n], gpu, tokens)
    tiles = 300 * top // K.routed_tile_rows(act, width, ff) + experts
    p = run_op(ops["moe_plan"], [r[2], i32(n, top), i32(experts + 1), i32(tiles, 4), i32(1), i32(1), n * top, i32(1)], gpu, tokens)
    there = p[1].view(-1)[p[1].view(-1) >= 0]
    assert sorted(there.tolist()) == list(range(len(there))) and torch.equal(p[1] < 0, r[2] >= experts) and int(p[7]) == 0
    g = run_op(ops["moe_gather"], [x, p[1], torch.zeros(300 * top, width, dtype=DT[act]), n * top], gpu, tokens)
    w1 = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)])
    w2 = torch.stack([w[f"e{e}.down"] for e in range(experts)])
    a = run_op(ops["moe_fc1"], [g[2], w1, torch.zeros(300 * top, ff, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)
    y = run_op(ops["moe_fc2"], [a[2], w2, torch.zeros(300 * top, width, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)
    sa = run_op(K.linear_op(2 * ff, width, act=act, epilogue="swiglu", rows_max=300), [x, torch.cat([w["shared.gate"], w["shared.up"]]),
                                                                                       torch.zeros(n, ff, dtype=DT[act]), n, i32(1)], gpu, tokens)
    sy = run_op(K.linear_op(width, ff, act=act, rows_max=300), [sa[2], w["shared.down"], torch.zeros(n, width, dtype=DT[act]), n, i32(1)], gpu, tokens)
    one, gate = bf(torch.ones(width)), torch.cat([logits.view(-1)[outputs:], torch.zeros(outputs)])      # the gate's column, as an argument with an offset sees it
    res = run_op(K.resid_scale_op(width, 1e-6, act, routed=top, shared_gate=outputs + 1, last=True),
                 [torch.zeros(n, width), y[2], one, torch.zeros(n, width), p[1], r[3], sy[2], gate, x], gpu, tokens)
    m = {"router": {"top": top, "experts": experts, "scale": 1.3, "groups": {"count": groups, "keep": keep}}}
    close(res[3], O.experts({k: v.double() for k, v in w.items()}, "", m, x.double()), act)


def prep(gpu, act, hq, hk, d, rot, halves, tied):
    """Norms over whole projections, rotation, keys and values into the cache; tied: the values are the keys as projected."""
    n, page, dt, pos_max = 6, 16, DT[act], 400
    v_col = hq * d if tied else (hq + hk) * d
    stride = (hq + 2 * hk) * d + 8
    qkv, pos, slots = rnd(n, stride, scale=3).to(dt), torch.tensor([0, 1, 399, 17, 64, 5]), torch.tensor([17, 0, -1, 47, 5, 16])
    qn, kn = bf(1 + rnd(hq * d, seed=1, scale=.4)), bf(1 + rnd(hk * d, seed=2, scale=.4))
    cache = torch.zeros(4 * hk * page * 2 * d * dt.itemsize, dtype=torch.uint8)
    base, factor = 300.0, 2.5
    tabs = run_op(C.rope_table_op(pos_max, rot, base, factor), [torch.zeros(pos_max, rot // 2), torch.zeros(pos_max, rot // 2)], gpu)
    op = K.qk_prep_whole_op(hq, hk, d, d, v_col, rot, page, stride, pos_max, 1e-4, act, halves)
    out = run_op(op, [qkv, cache, pos, slots, tabs[0], tabs[1], qn, kn, i32(1)], gpu, {"tokens": n})
    order = torch.arange(d)
    if not halves:      # the same rotation over columns in another order
        order[:rot] = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2)])

    def turn(x, w, heads):
        x = (O.rms(x.double(), 1e-4) * w.double()).reshape(n, heads, d)
        return O.rotate(x[..., order], pos, rot, base, factor)[..., torch.argsort(order)]

    close(out[0][:, : hq * d], turn(qkv[:, : hq * d], qn, hq).reshape(n, -1), act)
    assert torch.equal(out[0][:, hq * d:], qkv[:, hq * d:]) and int(out[8]) == 0
    pool = out[1].view(dt).view(4, hk * page * 2 * d)
    ks, vs = pool[:, : hk * page * d].view(4, hk, page, d), pool[:, hk * page * d:].view(4, hk, page, d)
    ok = slots >= 0
    close(ks[slots[ok] // page, :, slots[ok] % page], turn(qkv[:, hq * d:(hq + hk) * d], kn, hk)[ok], act)
    assert torch.equal(vs[slots[ok] // page, :, slots[ok] % page], qkv[:, v_col: v_col + hk * d].reshape(n, hk, d)[ok])
    rest = [i for i in range(64) if i not in slots.tolist()]
    assert not ks.transpose(1, 2).reshape(64, -1)[rest].any() and not vs.transpose(1, 2).reshape(64, -1)[rest].any()


def _paged(seqs, page, shape, dt, seed, scale=1.0):
    """Scattered pages of rows `shape` (heads first, columns last, or columns alone) -> (pages, table, rows of every sequence)."""
    width = 40
    pages = sum(-(-L // page) for L, _ in seqs) + 3
    order, at = torch.randperm(pages, generator=torch.Generator().manual_seed(3)).tolist(), 0
    *lead, cols = shape
    pool = rnd(pages, *lead, page, cols, seed=seed, scale=scale).to(dt)
    table = torch.zeros(len(seqs), width, dtype=torch.int32)
    for s, (L, _) in enumerate(seqs):
        for i in range(-(-L // page)):
            table[s, i] = order[at]
            at += 1
    flat = lambda t, s: torch.cat([t[table[s, i]] for i in range(-(-seqs[s][0] // page))], -2)[..., :seqs[s][0], :]
    return pool, table, flat


def _far_key(r, p, page):
    """The place of the key that stands far out for row r at position p, by turns: the first of all, a far one, the row's own, the
    last of the page before, the first of its page, the one after the row (another row's, which must not be seen)."""
    return max(0, [0, p // 3, p, p // page * page - 1, p // page * page, p + 1][r % 6])


def attention(gpu, act, hq, hk, d, dv, page, seqs, ragged, learned):
    """`seqs`: (context, new rows) of every sequence, over scattered pages. Most rows have a key that stands far out; every fifth
    turns away from all of them, so that the sink takes nearly everything."""
    dt, scale = DT[act], 0.35
    rows = [(s, L - R + i) for s, (L, R) in enumerate(seqs) for i in range(R)]
    n, gs, os_ = len(rows), hq * dv + 24, hq * dv + 8
    qs = hq * d + 16
    ks, table, flat = _paged(seqs, page, (hk, d), torch.float32, 4, .5)
    u = rnd(hk, d, seed=9)
    u = u / u.pow(2).sum(-1, keepdim=True).sqrt()
    ks = (ks + 2 * u[:, None]).to(dt)
    vs, _, _ = _paged(seqs, page, (hk, dv), dt, 5)
    sink = bf(2 + rnd(hq, seed=6, scale=2)) if learned else torch.zeros(hq)
    q = rnd(n, hq, d, seed=7, scale=.3)
    kf, vf = ([flat(t, s).transpose(0, 1).double() for s in range(len(seqs))] for t in (ks, vs))      # [L, hk, *]
    for r, (s, p) in enumerate(rows):
        for h in range(hq):
            c = kf[s][min(_far_key(r + h, p, page), seqs[s][0] - 1), h // (hq // hk)].float()
            q[r, h] += 12 * c / c.pow(2).sum() ** 0.5
            if (r + h) % 5 == 1:
                q[r, h] = -6 / scale * u[h // (hq // hk)]
    q = q.to(dt)
    buf, gate = torch.zeros(n, qs, dtype=dt), rnd(n, gs, seed=8, scale=2).to(dt)
    buf[:, : hq * d] = q.view(n, -1)
    pages = ks.shape[0]
    cache = torch.cat([ks.reshape(pages, -1), vs.reshape(pages, -1)], 1).contiguous().view(torch.uint8).view(-1)
    vars_, lens, extra = {"tokens": n, "seqs": len(seqs)}, ints([L for L, _ in seqs]), []
    if ragged and K.window_tiles(hq, hk, d, dv, page, act):
        cu = ints([0, *torch.tensor([R for _, R in seqs]).cumsum(0).tolist()])
        items = n // (64 // (hq // hk)) + len(seqs) + 1
        plan = run_op(C.attn_plan_op(hq, hk, len(seqs), d), [cu, i32(items, 2), i32(1), len(seqs), items, i32(len(seqs), 2), i32(1)], gpu, vars_)
        extra = [cu, plan[1], plan[2], plan[5], plan[6]]
    elif ragged:
        lens, extra = ints([p + 1 for _, p in rows]), [ints([s for s, _ in rows])]
    op = K.sink_attn_op(hq, hk, d, dv, scale, page, table.shape[1], qs, os_, gs, ragged, act, sink=learned, seqs_max=len(seqs))
    out = run_op(op, [buf, cache, torch.zeros(n, os_, dtype=dt), table, lens, gate, i32(1), *([sink] if learned else []), *extra], gpu, vars_)

    def wanted(r, sink):
        s, p = rows[r]
        o = O.attend(q[r:r + 1].double(), kf[s][:p + 1], vf[s][:p + 1], scale, sink.double())[0].reshape(-1)
        return o * O.sigmoid(gate[r, : hq * dv].double())

    want = torch.stack([wanted(r, sink) for r in range(n)])
    close(out[2][:, : hq * dv], want, act)
    assert not out[2][:, hq * dv:].any() and int(out[6]) == 0
    # without the sink some row is far away: the limit sees it
    assert max(float((wanted(r, sink - 1e4) - want[r]).abs().max() / want.abs().max()) for r in range(min(n, 8))) > 0.04


def latent_prep(gpu, act, rank, rot, q_rank):
    n, page, dt, pos_max, down = 5, 16, DT[act], 300, q_rank + rank + rot + 5
    x, pos, slots = rnd(n, down, scale=2).to(dt), torch.tensor([0, 299, 7, 64, 1]), torch.tensor([3, 40, -1, 0, 17])
    w, wq = bf(1 + rnd(rank, seed=1, scale=.3)), bf(1 + rnd(q_rank, seed=2, scale=.3))
    cache = torch.zeros(3 * page * (rank + rot) * dt.itemsize, dtype=torch.uint8)
    tabs = run_op(C.rope_table_op(pos_max, rot, 500.0), [torch.zeros(pos_max, rot // 2), torch.zeros(pos_max, rot // 2)], gpu)
    qs = q_rank + 2
    out = run_op(K.latent_prep_op(rank, rot, q_rank, down, qs, pos_max, 1e-4, act), [x, cache, torch.zeros(n, qs, dtype=dt), pos, slots, tabs[0], tabs[1], w, wq, i32(1)],
                 gpu, {"tokens": n})
    xd = x.double()
    close(out[2][:, :q_rank], O.rms(xd[:, :q_rank], 1e-4) * wq.double(), act)
    key = O.rotate(xd[:, None, q_rank + rank: q_rank + rank + rot], pos, rot, 500.0)[:, 0]
    want = torch.cat([O.rms(xd[:, q_rank: q_rank + rank], 1e-4) * w.double(), key], 1)
    got = out[1].view(dt).view(-1, rank + rot)
    close(got[slots[slots >= 0]], want[slots >= 0], act)
    assert not got[[i for i in range(3 * page) if i not in slots.tolist()]].any() and not out[2][:, q_rank:].any() and int(out[9]) == 0


def latent(gpu, act, H, rank, rot, page, seqs, ragged):
    """The absorbed form: rows [latent | turned key part], queries [absorbed | not yet turned], a sink per head."""
    dt, scale, base, pos_max = DT[act], 0.3, 200.0, 1200
    rows = [(s, L - R + i) for s, (L, R) in enumerate(seqs) for i in range(R)]
    n, rs = len(rows), H * rot + 8
    pool, table, flat = _paged(seqs, page, (rank + rot,), torch.float32, 4, .5)
    u, length = rnd(rank, seed=9), 2 * max(1.0, rank / 72) ** 0.5
    u = u / u.pow(2).sum().sqrt()
    pool[..., :rank] += length * u
    pool[..., rank:] *= (rank / rot) ** 0.5          # the turned part weighs as much as the latent
    pool = pool.to(dt)
    cf = [flat(pool, s).double() for s in range(len(seqs))]
    sink = bf(2 + rnd(H, seed=6, scale=2))
    ql, qr, pos = rnd(n, H, rank, seed=7, scale=.2), rnd(n, H, rot, seed=8, scale=.4), torch.tensor([p for _, p in rows])
    for r, (s, p) in enumerate(rows):
        for h in range(H):
            c = cf[s][min(_far_key(r + h, p, page), seqs[s][0] - 1)].float()
            size = c.pow(2).sum() ** 0.5
            ql[r, h] += (13 if (r + h) % 5 != 3 else 0) * c[:rank] / size      # some find their key by the turned part alone
            turned = c[None, None, rank:].double()
            qr[r, h] += 13 * O.rotate(turned, torch.tensor([-p]), rot, base)[0, 0].float() / size      # the row's turn brings it onto the key
            if (r + h) % 5 == 1:      # away from every key: the sink takes nearly everything
                ql[r, h], qr[r, h] = -12 / scale / length * u, 0
    ql, qr = ql.to(dt), qr.to(dt)
    tabs = run_op(C.rope_table_op(pos_max, rot, base), [torch.zeros(pos_max, rot // 2), torch.zeros(pos_max, rot // 2)], gpu)
    buf = torch.zeros(n, rs, dtype=dt)
    buf[:, : H * rot] = qr.view(n, -1)
    vars_ = {"tokens": n, "seqs": len(seqs)}
    lens, extra = (ints([p + 1 for _, p in rows]), [ints([s for s, _ in rows])]) if ragged else (ints([L for L, _ in seqs]), [])
    op = K.latent_rot_attn_op(H, rank, rot, scale, page, table.shape[1], pos_max, rs, ragged, act, seqs_max=len(seqs))
    out = run_op(op, [ql, pool.reshape(-1).view(torch.uint8), torch.zeros(n, H, rank, dtype=dt), table, lens, i32(1), *extra, buf, tabs[0], tabs[1], sink], gpu, vars_)
    turned = O.rotate(qr.double(), pos, rot, base)

    def wanted(r, sink, turned=turned):
        s, p = rows[r]
        q = torch.cat([ql[r].double(), turned[r]], -1)[None]
        return O.attend(q, cf[s][:p + 1, None], cf[s][:p + 1, None, :rank], scale, sink.double())[0]

    want = torch.stack([wanted(r, sink) for r in range(n)])
    close(out[2], want, act, 1.5)
    assert int(out[5]) == 0
    # without the sink, or the query's turn, some row is far away
    some = range(min(n, 12))
    for other in ([wanted(r, sink - 1e4) for r in some], [wanted(r, sink, qr.double()) for r in some]):
        assert float((torch.stack(other) - want[:len(other)]).abs().max() / want.abs().max()) > 0.06

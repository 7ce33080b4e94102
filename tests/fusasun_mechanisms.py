"""Each mechanism alone against its plain statement: bodies shared by the CPU and the GPU tests."""
import torch

from kern_b200.models import blocks as K
from kern_b200.models import common as C
from tests.gafapel_cases import run_op
from tests.gafapel_mechanisms import DT, bf, close, rnd
from tests.oracles import fusasun as O

i32 = lambda *s: torch.zeros(*s, dtype=torch.int32)
ints = lambda v: torch.tensor(v, dtype=torch.int32)


# ---- positions ----------------------------------------------------------------------------------------------------------
def _table(gpu, op, dims, frequencies, size, plain):
    """The tables turn a row of ones and zeros as the rotation does, also at far positions."""
    n, half = 4000, dims // 2
    out = run_op(op, [torch.zeros(n, half), torch.zeros(n, half)], gpu)
    x = torch.zeros(n, 1, dims).double()
    x[..., ::2] = 1
    want = O.rotate(x, torch.arange(n), frequencies, size)[:, 0]
    close(torch.stack([out[0], out[1]], -1).flatten(-2), want, "f32", 0.1)
    return float((O.rotate(x, torch.arange(n), plain)[:, 0] - want).abs().max())


def banded_table(gpu, dims, base, factor, low, high, original):
    s = {"factor": factor, "low": low, "high": high, "original": original}
    off = _table(gpu, C.rope_table_op(4000, dims, base, scaling=C.banded_rope(factor, low, high, original)), dims, O.banded_frequencies(dims, base, s), 1.0,
                 O.plain_frequencies(dims, base))
    assert off > 0.1 or factor == 1 or dims == 2


def yarn_table(gpu, dims, base, factor, original, fast, slow):
    f, size = O.yarn_frequencies(dims, base, {"factor": factor, "original": original, "fast": fast, "slow": slow})
    assert _table(gpu, C.rope_table_op(4000, dims, base, scaling=C.ramped_rope(dims, base, factor, original, fast, slow)), dims, f, size, O.plain_frequencies(dims, base)) > 0.05


# ---- the residual and what a mixer reads -----------------------------------------------------------------------------------
def _lines(width, taps, act, count, seed=0):
    """A state of `count` lines, and the rows each holds."""
    line = K.conv_line_bytes(width, taps, act)
    state, rows = torch.zeros(count * line, dtype=torch.uint8), rnd(count, taps - 1, width, seed=seed).to(DT[act])
    for i in range(count):
        part = rows[i].contiguous().view(-1).view(torch.uint8)
        state[i * line: i * line + part.numel()] = part
    return state, rows, line


def _kept(state, line, i, width, taps, act):
    return state[i * line: i * line + (taps - 1) * width * DT[act].itemsize].view(DT[act]).view(taps - 1, width)


def _check_conv(out, state, line, lines, rows, h, starts, w, width, taps, act, tol=1.0):
    """Every sequence's rows h against the oracle from the line it started with; line 0 gives zeros and keeps nothing."""
    for s, i in enumerate(lines):
        part = h[starts[s]: starts[s + 1]]
        st = {"h": rows[i].double() if i > 0 else torch.zeros(taps - 1, width).double()}
        if len(part):
            close(out[starts[s]: starts[s + 1]], O.input_conv(w.double(), part.double(), st), act, tol)
        if i > 0:
            assert torch.equal(_kept(state, line, i, width, taps, act).double(), st["h"])
    assert torch.equal(_kept(state, line, 0, width, taps, act), rows[0])


def embed(gpu, act, width, taps, scale):
    n, vocab = 5, 31
    ids, table, wn, w = torch.tensor([0, 30, 7, 7, 12]), bf(rnd(vocab, width)), bf(1 + rnd(width, seed=1, scale=.1)), bf(rnd(width, taps, seed=2, scale=.5))
    state, rows, line = _lines(width, taps, act, 7, 3)
    lines = [3, 0, 1, 6, 2]
    e = table[ids].double() * scale
    want = O.rms(e, 1e-4) * wn.double()
    new = lambda: [ids, table, wn, torch.zeros(n, width), torch.zeros(n, width, dtype=DT[act]), i32(1)]
    out = run_op(K.resid_embed_op(width, vocab, 1e-4, act, scale), new(), gpu, {"tokens": n})
    close(out[3], e, "f32")
    close(out[4], want, act)
    out = run_op(K.resid_embed_op(width, vocab, 1e-4, act, scale, (taps, line)), [*new(), w, torch.zeros(n, width, dtype=DT[act]), state, ints(lines)], gpu, {"tokens": n})
    close(out[3], e, "f32")
    close(out[4], want, act)
    _check_conv(out[7], out[8], line, lines, rows, out[4], range(n + 1), w, width, taps, act)
    assert int(out[5]) == 0


def conv_add(gpu, act, width, taps):
    """Sequences shorter and longer than the taps, one without rows, one on the line that is nobody's, and over borders of a thread's
    run of rows."""
    lens, lines = (1, 2, 33, 0, 5, 17, 1), [2, 5, 1, 4, 0, 3, 6]
    starts = [0, *torch.tensor(lens).cumsum(0).tolist()]
    n, w = starts[-1], bf(rnd(width, taps, seed=1, scale=.5))
    h = rnd(n, width, seed=2).to(DT[act])
    state, rows, line = _lines(width, taps, act, 7, 3)
    out = run_op(K.conv_add_op(width, taps, line, act), [h, w, torch.zeros(n, width, dtype=DT[act]), state, ints(lines), ints(starts), len(lens), n], gpu,
                 {"tokens": n, "seqs": len(lens)})
    _check_conv(out[2], out[3], line, lines, rows, h, starts, w, width, taps, act)


def resid_gate(gpu, act, width, routed, taps):
    """Gated, normed and added; `routed`: y holds as many expert rows per token. With the next input convolved, and as the last."""
    n, k, dt = 6, max(1, routed), DT[act]
    x, post, nxt, b = rnd(n, width), bf(1 + rnd(width, seed=1, scale=.3)), bf(1 + rnd(width, seed=2, scale=.3)), bf(rnd(width, seed=5, scale=2))
    y, gate, w = rnd(n * k, width, seed=3, scale=2).to(dt), rnd(n, width, seed=4, scale=3).to(dt), bf(rnd(width, taps, seed=9, scale=.5))
    perm, tw = torch.randperm(n * k, generator=torch.Generator().manual_seed(6)).int().view(n, k), rnd(n, k, seed=7).sigmoid()
    extra = [perm, tw] if routed else []
    v = (y.double()[perm.long()] * tw.double()[..., None]).sum(1) if routed else y.double()
    one = torch.eye(width).double()
    new = O.gated_sum(x.double(), v, gate.double(), one, b.double(), post.double(), 1e-4)      # the gate's product is given
    xn = torch.zeros(n, width, dtype=dt)
    out = run_op(K.resid_gate_op(width, 1e-4, act, routed), [x, y, post, nxt, xn, gate, b, *extra], gpu, {"tokens": n})
    close(out[0], new, "f32")
    close(out[4], O.rms(new, 1e-4) * nxt.double(), act)
    out = run_op(K.resid_gate_op(width, 1e-4, act, routed, last=True), [x, y, post, torch.zeros(n, width), gate, b, *extra], gpu, {"tokens": n})
    close(out[3], new, "f32")
    state, rows, line = _lines(width, taps, act, 8, 8)
    lines = [7, 2, 0, 4, 1, 3]
    out = run_op(K.resid_gate_op(width, 1e-4, act, routed, conv=(taps, line)), [x, y, post, nxt, xn, gate, b, *extra, w, torch.zeros(n, width, dtype=dt), state, ints(lines)],
                 gpu, {"tokens": n})
    close(out[0], new, "f32")
    close(out[4], O.rms(new, 1e-4) * nxt.double(), act)
    o = 7 + len(extra)
    _check_conv(out[o + 1], out[o + 2], line, lines, rows, out[4], range(n + 1), w, width, taps, act)


# ---- experts by table -----------------------------------------------------------------------------------------------------
def table_experts(gpu, act, width, ff, experts, top, n):
    vocab, tokens = 23, {"tokens": n}
    g = torch.Generator().manual_seed(1)
    table = torch.rand(vocab, experts, generator=g).argsort(-1)[:, :top].int().contiguous()
    ids, x = torch.randint(0, vocab, (n,), generator=g), rnd(n, width).to(DT[act])
    w = {f"e{e}.{t}": bf(rnd(r, c, seed=10 + e * 3 + len(t), scale=(2 if t != "down" else 1) * c ** -0.5))
         for e in range(experts) for t, (r, c) in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    r = run_op(K.route_table_op(experts, top, vocab), [ids, table, i32(n, top), torch.zeros(n, top), n, i32(1)], gpu, tokens)
    assert torch.equal(r[2], table[ids]) and int(r[5]) == 0
    ops = K.routed_ops(width, ff, experts, top, 300, act)
    tiles = 300 * top // K.routed_tile_rows(act, width, ff) + experts
    p = run_op(ops["moe_plan"], [r[2], i32(n, top), i32(experts + 1), i32(tiles, 4), i32(1), i32(1), n * top, i32(1)], gpu, tokens)
    rows = run_op(ops["moe_gather"], [x, p[1], torch.zeros(300 * top, width, dtype=DT[act]), n * top], gpu, tokens)[2]
    w1 = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)])
    w2 = torch.stack([w[f"e{e}.down"] for e in range(experts)])
    a = run_op(ops["moe_fc1"], [rows, w1, torch.zeros(300 * top, ff, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)
    y = run_op(ops["moe_fc2"], [a[2], w2, torch.zeros(300 * top, width, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)[2]
    got = (y.double()[p[1].long()] * r[3].double()[..., None]).sum(1)
    close(got, O.experts({k: v.double() for k, v in w.items()}, "", {"router": {"top": top}}, x.double(), ids, table), act)
    bad = run_op(K.route_table_op(experts, top, vocab), [torch.full((n,), vocab), table, i32(n, top), torch.zeros(n, top), n, i32(1)], gpu, tokens)
    assert int(bad[5]) != 0 and bool((bad[2] == -1).all())


# ---- attention ------------------------------------------------------------------------------------------------------------
def _pages_of(seqs, page, width=80):
    """Scattered pages for every sequence -> (table, number of pages)."""
    pages = sum(-(-L // page) for L, _ in seqs) + 3
    order, at, table = torch.randperm(pages, generator=torch.Generator().manual_seed(3)).tolist(), 0, i32(len(seqs), width)
    for s, (L, _) in enumerate(seqs):
        n = -(-L // page)
        table[s, :n] = ints(order[at: at + n])
        at += n
    return table, pages


def _place(pool_rows, table, s, page, rows):
    """rows [L, heads, cols] of sequence s into [pages, heads, page, cols]."""
    for j in range(rows.shape[0]):
        pool_rows[table[s, j // page], :, j % page] = rows[j]


def _block_place(b, pool, page):
    """(page of a sequence, slot in it) of block b: the page of the block's last token, and the count of earlier blocks that end there."""
    at = (b * pool + pool - 1) // page
    return at, sum(1 for e in range(b) if (e * pool + pool - 1) // page == at)


def _pool_cache(pages, z, hk, d, dv, act):
    """The second cache, filled with what must not be read -> (bytes, keys [pages, hk, slots, d], values)."""
    raw, n = torch.zeros(pages * z["page"], dtype=torch.uint8), hk * z["slots"] * (d + dv)
    rows = torch.as_strided(raw.view(DT[act]), (pages, n), (z["page"] // DT[act].itemsize, 1))
    rows.copy_(rnd(pages, n, seed=33, scale=3))
    return raw, rows[:, : hk * z["slots"] * d].unflatten(1, (hk, z["slots"], d)), rows[:, hk * z["slots"] * d:].unflatten(1, (hk, z["slots"], dv))


def prep(gpu, act, hq, hk, d, dv, rot, pool, page, L):
    """One sequence in portions (ragged calls, two tokens at least, and single rows): keys turned, values as they are, and the means of
    every block that has ended. A row without a slot leaves nothing."""
    dt, pos_max, stride = DT[act], 400, hq * d + hk * (d + dv) + 8
    z, (table, pages) = K.pooled_sizes(hk, d, dv, pool, page, act), _pages_of(((L, 1), (9, 1)), page)
    qkv = rnd(L, stride, scale=2).to(dt)
    cache = torch.zeros(pages * hk * page * (d + dv) * dt.itemsize, dtype=torch.uint8)
    pooled, pk, pv = _pool_cache(pages, z, hk, d, dv, act)
    before = (pk.clone(), pv.clone())
    tabs = run_op(C.rope_table_op(pos_max, rot, 300.0), [torch.zeros(pos_max, rot // 2), torch.zeros(pos_max, rot // 2)], gpu)
    slot = lambda p: int(table[0, p // page]) * page + p % page
    turned, lo, sizes, i = [], 0, (pool + 1, 2, 1, 1, 33, 1), 0
    while lo < L:
        n = min(sizes[i % len(sizes)], L - lo)
        i += 1
        part, pos, slots = qkv[lo: lo + n], torch.arange(lo, lo + n), torch.tensor([slot(p) for p in range(lo, lo + n)])
        if n > 1:      # a second sequence beside it, whose row has no slot and would end a block
            part, pos, slots = torch.cat([part, qkv[:1]]), torch.cat([pos, torch.tensor([pool - 1])]), torch.cat([slots, torch.tensor([-1])])
            op = K.qk_prep_pool_op(hq, hk, d, dv, rot, pool, page, table.shape[1], stride, pos_max, True, act)
            extra, vars_ = [ints([0, n, n + 1]), 2, n + 1], {"tokens": n + 1}
        else:
            op, extra, vars_ = K.qk_prep_pool_op(hq, hk, d, dv, rot, pool, page, table.shape[1], stride, pos_max, False, act), [], {"tokens": 1}
        out = run_op(op, [part, cache, pooled, pos, slots, table, tabs[0], tabs[1], i32(1), *extra], gpu, vars_)
        turned.append(out[0][:n])
        cache, pooled = out[1], out[2]
        assert int(out[8]) == 0
        lo += n
    f = O.plain_frequencies(rot, 300.0)
    q, k = (O.rotate(qkv[:, a: a + h * d].double().reshape(L, h, d), torch.arange(L), f) for a, h in ((0, hq), (hq * d, hk)))
    close(torch.cat(turned)[:, : hq * d], q.reshape(L, -1), act)
    rows = cache.view(dt).view(pages, -1)
    ks, vs = rows[:, : hk * page * d].view(pages, hk, page, d), rows[:, hk * page * d:].view(pages, hk, page, dv)
    at = torch.arange(L)
    held_k, held_v = ks[table[0, at // page].long(), :, at % page], vs[table[0, at // page].long(), :, at % page]
    close(held_k, k, act)
    assert torch.equal(held_v, qkv[:, (hq + hk) * d: hq * d + hk * (d + dv)].reshape(L, hk, dv))
    _, pk, pv = _pool_views(pooled, pages, z, hk, d, dv, dt)
    untouched = torch.ones(pages, z["slots"], dtype=torch.bool)
    for b in range(L // pool):
        pg, sl = _block_place(b, pool, page)
        untouched[table[0, pg], sl] = False
        part = slice(b * pool, b * pool + pool)
        close(pk[table[0, pg], :, sl], held_k[part].double().mean(0), act, 0.5)
        close(pv[table[0, pg], :, sl], held_v[part].double().mean(0), act, 0.5)
    for have, was in ((pk, before[0]), (pv, before[1])):
        assert torch.equal(have.transpose(1, 2)[untouched], was.transpose(1, 2)[untouched])


def _pool_views(raw, pages, z, hk, d, dv, dt):
    n = hk * z["slots"] * (d + dv)
    rows = torch.as_strided(raw.view(dt), (pages, n), (z["page"] // dt.itemsize, 1))
    return rows, rows[:, : hk * z["slots"] * d].unflatten(1, (hk, z["slots"], d)), rows[:, hk * z["slots"] * d:].unflatten(1, (hk, z["slots"], dv))


def _targets(p, window, pool, L):
    """Where a row at position p may be tempted to look: the edges of its window from both sides, the row after it, the last block it
    sees and the next one, the first block, and itself. ("key", position) or ("mean", block)."""
    seen = max(0, p - window + 1) // pool
    out = [("key", p), ("key", p - window + 1), ("key", p - window), ("key", p + 1), ("mean", seen - 1), ("mean", seen), ("mean", 0), ("key", seen * pool)]
    return [(kind, x) for kind, x in out if x >= 0 and (x < L if kind == "key" else (x + 1) * pool <= L)]


def attention(gpu, act, hq, hk, d, dv, window, pool, page, seqs, ragged):
    """`seqs`: (context, new rows) of every sequence over scattered pages. Every query points at one key or mean that stands out, some of
    them just outside what the row may see."""
    dt, scale = DT[act], 0.35
    rows = [(s, L - R + i) for s, (L, R) in enumerate(seqs) for i in range(R)]
    n, qs, os_ = len(rows), hq * d + 16, hq * dv + 8
    table, pages = _pages_of(seqs, page)
    z = K.pooled_sizes(hk, d, dv, pool, page, act)
    pooled, pk, pv = _pool_cache(pages, z, hk, d, dv, act)
    ks, vs = rnd(pages, hk, page, d, seed=21, scale=3).to(dt), rnd(pages, hk, page, dv, seed=22, scale=3).to(dt)
    kf, vf, km = [], [], []
    for s, (L, _) in enumerate(seqs):
        # tokens of a block lean to one side, so that means keep some length
        lean = rnd(-(-L // pool), hk, d, seed=40 + s).repeat_interleave(pool, 0)[:L]
        k, v = (rnd(L, hk, d, seed=4 + s, scale=.7) + .7 * lean).to(dt), rnd(L, hk, dv, seed=50 + s).to(dt)
        _place(ks, table, s, page, k)
        _place(vs, table, s, page, v)
        kf.append(k.double())
        vf.append(v.double())
        km.append(kf[s][: L // pool * pool].reshape(L // pool, pool, hk, d).mean(1))
        for b in range(L // pool):
            pg, sl = _block_place(b, pool, page)
            pk[table[s, pg], :, sl] = km[s][b].to(dt)
            pv[table[s, pg], :, sl] = vf[s][b * pool: b * pool + pool].mean(0).to(dt)
    q = rnd(n, hq, d, seed=7, scale=.3)
    for r, (s, p) in enumerate(rows):
        may = _targets(p, window, pool, seqs[s][0])
        for h in range(hq):
            kind, x = may[(r + h) % len(may)]
            c = (kf[s][x] if kind == "key" else km[s][x])[h // (hq // hk)].float()
            q[r, h] += 6 / scale * c / c.pow(2).sum()      # a score of about 6 there
    q = q.to(dt)
    buf = torch.zeros(n, qs, dtype=dt)
    buf[:, : hq * d] = q.view(n, -1)
    cache = torch.cat([ks.reshape(pages, -1), vs.reshape(pages, -1)], 1).contiguous().view(torch.uint8).view(-1)
    vars_, lens, extra = {"tokens": n, "seqs": len(seqs)}, ints([L for L, _ in seqs]), []
    if ragged and K.pooled_tiles(hq, hk, d, dv, pool, page, act):
        cu = ints([0, *torch.tensor([R for _, R in seqs]).cumsum(0).tolist()])
        items = n // (64 // (hq // hk)) + len(seqs) + 1
        plan = run_op(C.attn_plan_op(hq, hk, len(seqs), d), [cu, i32(items, 2), i32(1), len(seqs), items, i32(len(seqs), 2), i32(1)], gpu, vars_)
        extra = [cu, plan[1], plan[2], plan[5], plan[6]]
    elif ragged:
        lens, extra = ints([p + 1 for _, p in rows]), [ints([s for s, _ in rows])]
    op = K.pooled_attn_op(hq, hk, d, dv, window, pool, scale, page, table.shape[1], qs, os_, ragged, act, seqs_max=len(seqs))
    out = run_op(op, [buf, cache, pooled, torch.zeros(n, os_, dtype=dt), table, lens, i32(1), *extra], gpu, vars_)

    def wanted(r, window=window, pool=pool):
        s, p = rows[r]
        return O.pooled_window(q[r:r + 1].double(), O.heads_of(kf[s][:p + 1], hq), O.heads_of(vf[s][:p + 1], hq), scale, window, pool)[0].reshape(-1)

    want = torch.stack([wanted(r) for r in range(n)])
    close(out[3][:, : hq * dv], want, act, 1.5)
    assert not out[3][:, hq * dv:].any() and int(out[6]) == 0
    # a window one token off (of blocks of one token none is), or no pooled rows at all, is far away in some row
    late = [r for r in range(n) if rows[r][1] >= window + pool]
    for change in ({"window": window + 1}, {"window": max(1, window - 1)}, {"pool": 1 << 20}):
        if late and change.get("window") != window and (pool > 1 or "pool" in change):
            assert max(float((wanted(r, **change) - want[r]).abs().max()) for r in late[:12]) > 0.1 * float(want.abs().max()), change


def latent_prep(gpu, act, rank, rot, q_rank):
    n, page, dt, pos_max, down = 5, 16, DT[act], 300, q_rank + rank + rot + 5
    x, pos, slots = rnd(n, down, scale=2).to(dt), torch.tensor([0, 299, 7, 64, 1]), torch.tensor([3, 40, -1, 0, 17])
    w, wq = bf(1 + rnd(rank, seed=1, scale=.3)), bf(1 + rnd(q_rank, seed=2, scale=.3))
    cache = torch.zeros(3 * page * (rank + rot) * dt.itemsize, dtype=torch.uint8)
    f, size = O.yarn_frequencies(rot, 500.0, {"factor": 3.0, "original": 60, "fast": 8.0, "slow": 1.0})
    tabs = run_op(C.rope_table_op(pos_max, rot, 500.0, scaling=C.ramped_rope(rot, 500.0, 3.0, 60, 8.0, 1.0)), [torch.zeros(pos_max, rot // 2), torch.zeros(pos_max, rot // 2)], gpu)
    op = K.latent_prep_op(rank, rot, q_rank, down, q_rank, pos_max, 1e-4, act, halves=False)
    out = run_op(op, [x, cache, torch.zeros(n, q_rank, dtype=dt), pos, slots, tabs[0], tabs[1], w, wq, i32(1)], gpu, {"tokens": n})
    xd = x.double()
    close(out[2], O.rms(xd[:, :q_rank], 1e-4) * wq.double(), act)
    key = O.rotate(xd[:, None, q_rank + rank: q_rank + rank + rot], pos, f, size)[:, 0]
    want = torch.cat([O.rms(xd[:, q_rank: q_rank + rank], 1e-4) * w.double(), key], 1)
    got = out[1].view(dt).view(-1, rank + rot)
    close(got[slots[slots >= 0]], want[slots >= 0], act)
    assert not got[[i for i in range(3 * page) if i not in slots.tolist()]].any() and int(out[9]) == 0


def latent(gpu, act, H, rank, rot, window, page, seqs, ragged):
    """The absorbed form in a window: rows [latent | turned key part], queries [absorbed | not yet turned], a gate per head. Queries point
    at the edges of the window from both sides, some by the turned part alone."""
    dt, scale, base, pos_max, factor = DT[act], 0.3, 200.0, 1200, 2.0
    rows = [(s, L - R + i) for s, (L, R) in enumerate(seqs) for i in range(R)]
    n, rs, gs = len(rows), H * rot + 8, H + 5
    table, pages = _pages_of(seqs, page)
    pool, cf = rnd(pages, 1, page, rank + rot, seed=4, scale=3).to(dt), []
    for s, (L, _) in enumerate(seqs):
        c = rnd(L, 1, rank + rot, seed=60 + s, scale=.5)
        c[..., rank:] *= (rank / rot) ** 0.5          # the turned part weighs as much as the latent
        _place(pool, table, s, page, c.to(dt))
        cf.append(c[:, 0].to(dt).double())
    f, size = O.yarn_frequencies(rot, base, {"factor": factor, "original": 100, "fast": 10.0, "slow": 1.0})
    ql, qr, pos = rnd(n, H, rank, seed=7, scale=.2), rnd(n, H, rot, seed=8, scale=.4), torch.tensor([p for _, p in rows])
    for r, (s, p) in enumerate(rows):
        may = [x for x in (p, p - window + 1, p - window, p + 1, 0, p // page * page) if 0 <= x < seqs[s][0]]
        for h in range(H):
            c = cf[s][may[(r + h) % len(may)]].float()
            pull = 6 / scale / c.pow(2).sum()
            ql[r, h] += (2 * pull if (r + h) % 5 != 3 else 0) * c[:rank]
            back = O.rotate(c[None, None, rank:].double(), torch.tensor([-p]), f)[0, 0].float() / size      # the row's turn brings it onto the key
            qr[r, h] += 2 * pull * back
    ql, qr = ql.to(dt), qr.to(dt)
    tabs = run_op(C.rope_table_op(pos_max, rot, base, scaling=C.ramped_rope(rot, base, factor, 100, 10.0, 1.0)),
                  [torch.zeros(pos_max, rot // 2), torch.zeros(pos_max, rot // 2)], gpu)
    buf, gate = torch.zeros(n, rs, dtype=dt), rnd(n, gs, seed=9, scale=2).to(dt)
    buf[:, : H * rot] = qr.view(n, -1)
    vars_ = {"tokens": n, "seqs": len(seqs)}
    lens, extra = (ints([p + 1 for _, p in rows]), [ints([s for s, _ in rows])]) if ragged else (ints([L for L, _ in seqs]), [])
    op = K.latent_rot_attn_op(H, rank, rot, scale, page, table.shape[1], pos_max, rs, ragged, act, seqs_max=len(seqs), sink=False, halves=False, window=window, gate_stride=gs)
    out = run_op(op, [ql, pool.reshape(-1).view(torch.uint8), torch.zeros(n, H, rank, dtype=dt), table, lens, i32(1), *extra, buf, tabs[0], tabs[1], gate], gpu, vars_)
    turned = O.rotate(qr.double(), pos, f, size)

    def wanted(r, window=window, turned=turned):
        s, p = rows[r]
        q = torch.cat([ql[r].double(), turned[r]], -1)[None]
        c = cf[s][:p + 1, None].expand(-1, H, -1)
        return O.window(q, c, c[..., :rank], scale, window)[0] * O.sigmoid(gate[r, :H].double())[:, None]

    want = torch.stack([wanted(r) for r in range(n)])
    close(out[2], want, act, 1.5)
    assert int(out[5]) == 0
    late = [r for r in range(n) if rows[r][1] >= window][:12]
    for change in ({"window": window + 1}, {"window": max(1, window - 1)}, {"turned": qr.double()}):
        if late and change.get("window") != window and (window > 1 or "turned" not in change):      # one key alone takes everything
            assert max(float((wanted(r, **change) - want[r]).abs().max()) for r in late) > 0.05 * float(want.abs().max()), change

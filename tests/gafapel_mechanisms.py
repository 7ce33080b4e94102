"""Each mechanism alone against its plain statement: bodies shared by the CPU and the GPU tests."""
import torch

from kern_b200.models import blocks as K
from kern_b200.models import common as C
from tests.gafapel_cases import run_op
from tests.oracles import gafapel as O

DT = {"bf16": torch.bfloat16, "f32": torch.float32}
TOL = {"bf16": 2e-2, "f32": 2e-5}


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def bf(t):
    return t.to(torch.bfloat16)


def close(got, want, act, factor=1.0):
    want = want.double()
    err = float((got.double() - want).abs().max() / want.abs().max().clamp_min(1e-6))
    assert err < TOL[act] * factor, err


def embed(gpu, act, width, streams):
    n, vocab, pos = 7, 31, 19
    ids, at = torch.arange(n) * 3 % vocab, torch.tensor([0, 5, 18, 1, 2, 7, 3])
    table, ptab, we = bf(rnd(vocab, width)), bf(rnd(pos, width, seed=1)), bf(1 + rnd(width, seed=2, scale=.1))
    win, wn = bf(rnd(streams, seed=3)), bf(1 + rnd(width, seed=4, scale=.1))
    op = K.hyper_embed_op(width, streams, vocab, pos, 1e-5, act)
    out = run_op(op, [ids, at, table, ptab, we, win, wn, torch.zeros(n, streams, width), torch.zeros(n, width, dtype=DT[act]),
                      torch.zeros(1, dtype=torch.int32)], gpu, {"tokens": n})
    w = {"embed": table.double(), "pos": ptab.double(), "embed.norm": we.double()}
    e = O.embed(w, ids, at, 1e-5)
    close(out[7], e[:, None].repeat(1, streams, 1), "f32")
    close(out[8], O.rms(O.hyper_in(e[:, None].repeat(1, streams, 1), win.double()), 1e-5) * wn.double(), act)
    assert int(out[9]) == 0


def hyper(gpu, act, width, streams, routed):
    n, k = 6, max(1, routed)
    x, mix, wo = rnd(n, streams, width), bf(rnd(streams, streams, seed=1)), bf(rnd(streams, seed=2))
    win, wn = bf(rnd(streams, seed=3)), bf(1 + rnd(width, seed=4, scale=.1))
    y = rnd(n * k, width, seed=5).to(DT[act])
    perm = torch.randperm(n * k, generator=torch.Generator().manual_seed(6)).int()
    tw = torch.softmax(rnd(n, k, seed=7), -1)
    extra = [perm, tw] if routed else []
    yv = (y[perm.long()].double().view(n, k, width) * tw.double()[..., None]).sum(1) if routed else y.double()
    new = O.hyper_out(x.double(), yv, mix.double(), wo.double())
    out = run_op(K.hyper_mix_op(width, streams, 1e-6, act, routed), [x, y, mix, wo, win, wn, torch.zeros(n, width, dtype=DT[act]), *extra], gpu, {"tokens": n})
    close(out[0], new, "f32")
    close(out[6], O.rms(O.hyper_in(new, win.double()), 1e-6) * wn.double(), act)
    out = run_op(K.hyper_last_op(width, streams, act, routed), [x, y, mix, wo, torch.zeros(n, width), *extra], gpu, {"tokens": n})
    close(out[4], new.sum(1), "f32", 3)


def row_norm(gpu, act):
    src, w = rnd(9, 40), bf(1 + rnd(40, seed=1, scale=.1))
    rows, cu = torch.tensor([8, 0, 3, 3], dtype=torch.int32), torch.tensor([0, 2, 3, 9], dtype=torch.int32)
    want = O.rms(src.double(), 1e-6) * w.double()
    y = lambda n: torch.zeros(n, 40, dtype=DT[act])
    close(run_op(K.row_norm_op(40, 1e-6, 9, act, "listed"), [src, w, y(4), rows], gpu, {"wanted": 4})[2], want[rows.long()], act)
    close(run_op(K.row_norm_op(40, 1e-6, 9, act, "last"), [src, w, y(3), cu], gpu, {"seqs": 3})[2], want[[1, 2, 8]], act)
    close(run_op(K.row_norm_op(40, 1e-6, 9, act, "each"), [src, w, y(5)], gpu, {"seqs": 5})[2], want[:5], act)


def linear(gpu, act, m, n, k, epilogue):
    a, w = rnd(m, k).to(DT[act]), bf(rnd((2 if epilogue == "swiglu" else 1) * n, k, seed=1, scale=k ** -0.5))
    want = a.double() @ w.double().t()
    if epilogue == "swiglu":
        want = O.silu(want[:, :n]) * want[:, n:]
    c = torch.zeros(m, n, dtype=torch.float32 if epilogue == "f32" else DT[act])
    op = K.linear_op(2 * n if epilogue == "swiglu" else n, k, act=act, epilogue=epilogue, rows_max=max(m, 300))
    out = run_op(op, [a, w, c, m, torch.zeros(1, dtype=torch.int32)], gpu, {"tokens": m})
    close(out[2], want, act)
    assert int(out[4]) == 0


def head_linear(gpu, act, m, heads, n, k, transposed):
    lda = heads * k + 8
    a, w = rnd(m, lda).to(DT[act]), bf(rnd(heads, n, k, seed=1, scale=k ** -0.5))
    want = torch.cat([a[:, h * k:(h + 1) * k].double() @ w[h].double().t() for h in range(heads)], 1)
    src = w.transpose(1, 2).contiguous() if transposed else w
    op = K.head_linear_op(heads, n, k, act=act, rows_max=max(m, 300), lda=lda, ldc=heads * n, transposed=transposed)
    out = run_op(op, [a, src, torch.zeros(m, heads * n, dtype=DT[act]), m, torch.zeros(1, dtype=torch.int32)], gpu, {"tokens": m})
    close(out[2], want, act)
    assert int(out[4]) == 0


def transpose(gpu):
    w = bf(rnd(3, 37, 50))
    assert torch.equal(run_op(K.transpose_heads_op(3, 37, 50), [w, torch.zeros(3, 50, 37, dtype=torch.bfloat16)], gpu)[1], w.transpose(1, 2))


def gate(gpu, act):
    x, g = rnd(11, 24).to(DT[act]), rnd(11, 30, seed=1, scale=3).to(DT[act])
    out = run_op(K.gate_mul_op(24, 30, act), [x, g, torch.zeros(11, 24, dtype=DT[act]), 11], gpu, {"tokens": 11})
    close(out[2], x.double() / (1 + torch.exp(-g[:, :24].double())), act)


def route(gpu):
    z, b = rnd(13, 40, scale=2), bf(rnd(40, seed=1, scale=2))
    out = run_op(K.route_logits_op(40, 5), [z, b, torch.zeros(13, 5, dtype=torch.int32), torch.zeros(13, 5), 13], gpu, {"tokens": 13})
    for t, chosen in enumerate(O.route(z.double() + b.double(), 5)):
        assert [e for e, _ in chosen] == out[2][t].tolist()
        close(out[3][t], torch.stack([v for _, v in chosen]), "f32")


def routed_experts(gpu, act, width, ff, experts, top, n):
    """Router to combined rows, and a bias that decides: an expert no logit favours takes every token."""
    x = rnd(n, width).to(DT[act])
    wr, br = bf(rnd(experts, width, seed=1, scale=2 * width ** -0.5)), bf(rnd(experts, seed=2))
    br[experts - 1] = 30.0
    w = {"router": wr, "router.b": br}
    for e in range(experts):
        for t, (r, c) in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            w[f"e{e}.{t}"] = bf(rnd(r, c, seed=10 + e * 3 + len(t), scale=c ** -0.5))
    ops, tokens = K.routed_ops(width, ff, experts, top, 300, act), {"tokens": n}
    i32 = lambda *s: torch.zeros(*s, dtype=torch.int32)
    logits = (x.float() @ wr.float().t())
    r = run_op(K.route_logits_op(experts, top), [logits, br, i32(n, top), torch.zeros(n, top), n], gpu, tokens)
    assert (r[2] == experts - 1).any(1).all()
    tiles = 300 * top // K.routed_tile_rows(act, width, ff) + experts
    p = run_op(ops["moe_plan"], [r[2], i32(n, top), i32(experts + 1), i32(tiles, 4), i32(1), i32(1), n * top, i32(1)], gpu, tokens)
    assert sorted(p[1].view(-1).tolist()) == list(range(n * top)) and int(p[7]) == 0
    g = run_op(ops["moe_gather"], [x, p[1], torch.zeros(300 * top, width, dtype=DT[act]), n * top], gpu, tokens)
    w1 = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)])
    w2 = torch.stack([w[f"e{e}.down"] for e in range(experts)])
    a = run_op(ops["moe_fc1"], [g[2], w1, torch.zeros(300 * top, ff, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)
    y = run_op(ops["moe_fc2"], [a[2], w2, torch.zeros(300 * top, width, dtype=DT[act]), p[3], p[4], n * top, i32(1)], gpu, tokens)
    got = (y[2][p[1].long()].float() * r[3][..., None]).sum(1)
    want = O.experts({k: v.double() for k, v in w.items()}, "", {"router": {"top": top}}, x.double())
    close(got, want, act)


def conv_and_state(gpu, act, ch, taps, chunks, ragged):
    """Three sequences (one on the null line never asked about) in chunks against whole ones; windows end as the history."""
    lens = [sum(c) for c in chunks]
    stride, dt = ch + 4, DT[act]
    u = [rnd(n, ch, seed=i).to(dt) for i, n in enumerate(lens)]
    w, b = bf(rnd(ch, taps, seed=20)), bf(rnd(ch, seed=21))
    line = ((taps - 1) * ch * dt.itemsize + 255) // 256 * 256 + 256
    state = torch.zeros(5 * line, dtype=torch.uint8)
    lines = torch.tensor([3, 1, 4], dtype=torch.int32)
    want = [O.short_conv(x.double(), torch.zeros(taps - 1, ch, dtype=torch.float64), w.double(), b.double()) for x in u]
    at = [0, 0, 0]
    op = K.short_conv_op(ch, taps, stride, line, ragged, act)
    for step in zip(*chunks):
        rows = torch.cat([u[i][at[i]:at[i] + n] for i, n in enumerate(step)])
        x = torch.zeros(len(rows), stride, dtype=dt)
        x[:, :ch] = rows
        cu = torch.tensor([0, *torch.tensor(step).cumsum(0).tolist()], dtype=torch.int32)
        y = torch.zeros(len(rows), ch, dtype=dt)
        out = run_op(op, [x, y, state, lines, *([cu] if ragged else []), w, b, 3, len(rows)], gpu, {"tokens": len(rows), "seqs": 3})
        state = out[2]
        close(out[1], torch.cat([want[i][0][at[i]:at[i] + n] for i, n in enumerate(step)]), act)
        at = [a + n for a, n in zip(at, step)]
    for i, ln in enumerate(lines.tolist()):
        win = state[ln * line: ln * line + (taps - 1) * ch * dt.itemsize].view(dt).view(taps - 1, ch)
        assert torch.equal(win.double(), want[i][1])
    assert int(state[:line].sum()) == 0 and int(state[2 * line:3 * line].sum()) == 0


def ssd(gpu, act, H, P, N, G, chunks, ragged):
    lens = [sum(c) for c in chunks]
    inner, ch, dt = H * P, H * P + 2 * G * N, DT[act]
    xbc = [rnd(n, ch, seed=i).to(dt) for i, n in enumerate(lens)]
    raw = [(rnd(n, H, seed=10 + i) - 1).to(dt) for i, n in enumerate(lens)]
    A, bias, D = bf(rnd(H, seed=20)), bf(rnd(H, seed=21)), bf(rnd(H, seed=22))
    want = []
    for i in range(2):
        r = xbc[i].double()
        want.append(O.state_space(r[:, :inner].reshape(-1, H, P), r[:, inner:inner + G * N].reshape(-1, G, N),
                                  r[:, inner + G * N:].reshape(-1, G, N), raw[i].double(), A.double(), bias.double(), D.double(),
                                  torch.zeros(H, N, P, dtype=torch.float64), G))
    s_off, stride = 256, H + 3
    line = 256 + (H * P * N * 4 + 255) // 256 * 256
    state, lines, at = torch.zeros(4 * line, dtype=torch.uint8), torch.tensor([3, 1], dtype=torch.int32), [0, 0]
    op = K.ssd_rule_op(H, P, N, G, stride, line, s_off, ragged, act)
    for step in zip(*chunks):
        n = sum(step)
        x = torch.cat([xbc[i][at[i]:at[i] + k] for i, k in enumerate(step)])
        d = torch.zeros(n, stride, dtype=dt)
        d[:, :H] = torch.cat([raw[i][at[i]:at[i] + k] for i, k in enumerate(step)])
        cu = torch.tensor([0, step[0], n], dtype=torch.int32)
        out = run_op(op, [x, d, torch.zeros(n, inner), state, lines, *([cu] if ragged else []), A, bias, D, 2], gpu, {"tokens": n, "seqs": 2})
        state = out[3]
        close(out[2], torch.cat([want[i][0][at[i]:at[i] + k].reshape(k, inner) for i, k in enumerate(step)]), "f32", 5)
        at = [a + k for a, k in zip(at, step)]
    for i, ln in enumerate(lines.tolist()):
        S = state[ln * line + s_off: ln * line + s_off + H * P * N * 4].view(torch.float32).view(H, P, N)
        close(S, want[i][1].transpose(1, 2), "f32", 5)
    assert int(state[:line].sum()) == 0 and int(state[2 * line:3 * line].sum()) == 0


def gate_norm(gpu, act, inner, parts):
    y, z, w = rnd(5, inner), rnd(5, inner + 8, seed=1).to(DT[act]), bf(1 + rnd(inner, seed=2, scale=.1))
    out = run_op(K.ssd_gate_norm_op(inner, parts, inner + 8, 1e-5, act), [y, z, w, torch.zeros(5, inner, dtype=DT[act])], gpu, {"tokens": 5})
    close(out[3], O.gated_group_norm(y.double(), z[:, :inner].double(), w.double(), parts, 1e-5), act)


def append(gpu, act, rank):
    lat, w = rnd(6, rank + 8).to(DT[act]), bf(1 + rnd(rank, seed=1, scale=.1))
    slots = torch.tensor([17, 0, -1, 31, 5, 16])
    cache = torch.zeros(32 * rank * DT[act].itemsize, dtype=torch.uint8)
    out = run_op(K.latent_append_op(rank, rank + 8, 1e-6, act), [lat, cache, slots, w], gpu, {"tokens": 6})
    got, ok = out[1].view(DT[act]).view(32, rank), slots >= 0
    close(got[slots[ok]], (O.rms(lat[:, :rank].double(), 1e-6) * w.double())[ok], act)
    rest = [i for i in range(32) if i not in slots.tolist()]
    assert not got[rest].any()


def attention(gpu, act, heads, rank, page, lens, ragged, seqs_max=8):
    """Rows against scattered pages. One key per row stands far out (its place walks from the first token over page borders
    to the row's own position), so a key that is missed, or one beyond the row's reach that is seen, decides the result."""
    table_width = 40
    dt = DT[act]
    pages = sum(-(-n // page) for n in lens) + 3
    order = torch.randperm(pages, generator=torch.Generator().manual_seed(3)).tolist()
    cache = rnd(pages, page, rank, seed=4, scale=.5).to(dt)
    table, at = torch.zeros(len(lens), table_width, dtype=torch.int32), 0
    for s, n in enumerate(lens):
        for i in range(-(-n // page)):
            table[s, i] = order[at]
            at += 1
    if ragged:
        rows = [(s, p) for s, n in enumerate(lens) for p in sorted({0, 1, page - 1, page, n // 2, n - 2, n - 1} & set(range(n)))]
    else:
        rows = [(s, n - 1) for s, n in enumerate(lens)]
    q = rnd(len(rows), heads, rank, seed=5, scale=.3)
    flat = lambda s: torch.cat([cache[table[s, i]] for i in range(-(-lens[s] // page))])
    for r, (s, p) in enumerate(rows):
        for h in range(heads):
            key = [0, page - 1, page, p - 1, p, p // 2][(r + h) % 6]
            key = min(max(key, 0), p)
            c = flat(s)[key].float()
            q[r, h] += 12 * c / c.pow(2).sum() ** 0.5
    # keys past a row's reach that would win if they were seen
    q = q.to(dt)
    row_seq = torch.tensor([s for s, _ in rows], dtype=torch.int32)
    row_len = torch.tensor([p + 1 for _, p in rows], dtype=torch.int32)
    op = K.latent_attn_op(heads, rank, 0.7, page, table_width, ragged, act, seqs_max=seqs_max)
    out = run_op(op, [q.view(len(rows), -1), cache.view(torch.uint8).view(-1), torch.zeros(len(rows), heads * rank, dtype=dt), table, row_len,
                      torch.zeros(1, dtype=torch.int32), *([row_seq] if ragged else [])], gpu, {"tokens": len(rows), "seqs": len(rows)})
    want = []
    for r, (s, p) in enumerate(rows):
        c = flat(s)[:p + 1].double()[:, None].expand(-1, heads, -1)
        want.append(O.attend(q[r:r + 1].double(), c, c, 0.7)[0].reshape(-1))
    close(out[2], torch.stack(want), act)
    assert int(out[5]) == 0

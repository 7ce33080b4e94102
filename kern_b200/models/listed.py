"""What the manifests of decoders with listed layers share: config.json names every layer with its mixer and feed-forward, a
program walks the list, the residual is f32, and the last sublayer leaves its rows in `hidden` (a carry: the rows of the last
call), from which `prefill` / `decode` norm and project each sequence's last row and the `logits` program any listed rows.

`Listed` collects buffers, ops, states and load-time calls while a family writes its sublayers; every op and weight is made
once, under a name that says its sizes.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

from . import blocks as K
from . import common as C

WANTED = 512          # most rows one call of the `logits` program projects


class Listed:
    def __init__(self, cfg):
        """`cfg`: width, vocab, eps, dtype, max_tokens, max_seqs, context, table_width, page_size, sampling, name."""
        if cfg.dtype not in K.ACT_BYTES:
            raise ValueError(f"dtype `{cfg.dtype}`: bf16 or f32")
        if not cfg.depth:
            raise ValueError("a model without layers")
        self.cfg, self.act, self.es = cfg, cfg.dtype, K.ACT_BYTES[cfg.dtype]
        self.bufs, self.ops, self.states, self.once = {}, {}, {}, []
        self.plans = {}      # name -> (buffers, op, args): what a ragged call's attention needs, made with the embedding
        self.err = self.B("error")

    # ---- names ----
    @staticmethod
    def B(name: str, offset: int = 0) -> dict:
        return {"buf": name, "offset": offset} if offset else {"buf": name}

    @staticmethod
    def V(name: str) -> dict:
        return {"var": name}

    def op(self, name: str, make) -> str:
        """An op under a name that says its sizes, made once."""
        if name not in self.ops:
            self.ops[name] = make()
        return name

    def room(self, name: str, cols: int, dtype: str | None = None, kind: str = "workspace") -> None:
        """A per-token buffer as wide as the widest layer that uses it."""
        have = self.bufs.get(name, {"shape": ["tokens", 0]})["shape"][1]
        self.bufs[name] = {"dtype": dtype or self.act, "shape": ["tokens", max(have, cols)], "kind": kind}

    def weight(self, name: str, shape, *tensors, dtype: str = "bf16") -> dict:
        if name not in self.bufs:
            self.bufs[name] = {"dtype": dtype, "shape": list(shape), "kind": "weight",
                               "bind": [t if isinstance(t, dict) else {"tensor": t} for t in tensors]}
        return self.B(name)

    def same(self, name: str, shape, dtype: str = "bf16") -> dict:
        return self.weight("w." + name, shape, name, dtype=dtype)

    def rows_weight(self, name: str, width: int, parts: list[tuple[str, int]]) -> tuple[dict, int]:
        """Projections with one input as one matrix -> (the weight, its rows), filled up to whole 16-byte vectors of output with
        copies of the first rows, which nobody reads. `parts`: (tensor, rows)."""
        rows = sum(n for _, n in parts)
        proj = -(-rows // 8) * 8
        (first, n), fill, left = parts[0], [], proj - rows
        while left > 0:
            fill.append({"tensor": first, "rows": [0, min(n, left)]})
            left -= n
        return self.weight(name, (proj, width), *[t for t, _ in parts], *fill), proj

    def linear(self, base: str, n: int, k: int, a, w, c, rows: str = "tokens", label: str = "", bias: dict | None = None, **kw) -> dict:
        kw |= {"bias": True} if bias else {}
        most = {"tokens": self.cfg.max_tokens, "seqs": self.cfg.max_seqs, "wanted": WANTED}[rows]
        lda = kw.get("lda")
        name = self.op(f"{base}_{n}x{k}" + (f"_of{lda}" if lda else ""), lambda: K.linear_op(n, k, act=self.act, rows_var=rows, rows_max=most, **kw))
        return {"op": name, "label": label, "args": [a, w, c, self.V(rows), self.err, *([bias] if bias else [])]}

    # ---- inputs and outputs ----
    def inputs(self, paged: str | None, lined: str | None, positions: bool = True, row_plan: bool = True) -> None:
        """The host's columns. `paged` / `lined`: a paged and a per-sequence state, when the model has them; `positions`: whether
        anything reads them; `row_plan`: room for every token's table row and reach (`rows_call`)."""
        cfg, S = self.cfg, self.cfg.max_seqs
        inp = lambda dt, shape, **kw: {"dtype": dt, "shape": shape, "kind": "input", **kw}
        self.bufs["token_ids"] = inp("i64", ["tokens"], fill="token", domain={"min": 0, "max": cfg.vocab - 1})
        if positions:
            self.bufs["positions"] = inp("i64", ["tokens"], fill="position", domain={"min": 0, "max": cfg.context - 1})
        self.bufs["cu_seqlens"] = inp("i32", [S + 1], fill="cu_seqlens")
        if paged:
            self.bufs["slot_mapping"] = inp("i64", ["tokens"], fill="slot", domain={"index_into": paged})
            self.bufs["seq_lens"] = inp("i32", ["seqs"], fill="seq_len")
            self.bufs["block_table"] = inp("i32", ["seqs", cfg.table_width], domain={"index_into": paged, "stride": cfg.page_size})
            if row_plan:
                self.bufs["row_seq"] = {"dtype": "i32", "shape": ["tokens"], "kind": "workspace"}
                self.bufs["row_len"] = {"dtype": "i32", "shape": ["tokens"], "kind": "workspace"}
        if lined:
            self.bufs["lines"] = inp("i32", [1, "seqs"], domain={"index_into": lined})
        self.bufs["next_token"] = {"dtype": "i64", "shape": ["seqs"], "kind": "output", "fill": "tokens"}
        self.bufs["error"] = {"dtype": "i32", "shape": [1], "kind": "output", "fill": "error"}

    def outputs(self) -> None:
        cfg, d = self.cfg, self.cfg.width
        self.room("hidden", d, "f32", "carry")
        self.bufs["last_n"] = {"dtype": self.act, "shape": ["seqs", d], "kind": "workspace"}
        self.bufs["logits"] = {"dtype": "f32", "shape": ["seqs", cfg.vocab], "kind": "workspace"}
        self.bufs["want_rows"] = {"dtype": "i32", "shape": ["wanted"], "kind": "input"}
        self.bufs["want_n"] = {"dtype": self.act, "shape": ["wanted", d], "kind": "workspace"}
        self.bufs["want_logits"] = {"dtype": "f32", "shape": ["wanted", cfg.vocab], "kind": "output"}

    def rows_call(self, label: str) -> dict:
        """The plan of a ragged call for kernels that take one attention row per token."""
        B, V = self.B, self.V
        return {"op": self.op("rows", C.mla_rows_op), "label": label,
                "args": [B("positions"), B("cu_seqlens"), B("row_seq"), B("row_len"), V("seqs"), V("tokens")]}

    # ---- the first call, and what rides with it ----
    def rotary(self, dims: int, base: float, factor: float = 1.0, scaling: dict | None = None) -> list[dict]:
        """The cos and sin tables of one rotation, written when the model is loaded; `scaling` as `rope_table_op` takes it."""
        context, B = self.cfg.context, self.B
        tag = f"{dims}x{base!r}" + (f"x{factor!r}" if factor != 1.0 else "") + ("_".join(["", scaling["kind"], *map(repr, scaling["constants"])]) if scaling else "")
        name = "rope." + tag
        if name + ".cos" not in self.bufs:
            for n in (".cos", ".sin"):
                self.bufs[name + n] = {"dtype": "f32", "shape": [context, dims // 2], "kind": "carry"}
            op = self.op("rope_" + tag, lambda: C.rope_table_op(context, dims, base, factor, scaling))
            self.once.append({"op": op, "label": name, "args": [B(name + ".cos"), B(name + ".sin")]})
        return [B(name + ".cos"), B(name + ".sin")]

    def lists_of(self, hq: int, hk: int, dim: int) -> list[dict]:
        """The work lists of a tensor-core attention; layers whose blocks hold as many tokens share them."""
        cfg, B = self.cfg, self.B
        name = f"plan.{hq // hk}" + (".128" if dim == 128 else "")
        if name not in self.plans:
            items = cfg.max_tokens // (64 // (hq // hk)) + cfg.max_seqs + 1
            for n, shape in ((".work_p", [items, 2]), (".count_p", [1]), (".work_d", [cfg.max_seqs, 2]), (".count_d", [1])):
                self.bufs[name + n] = {"dtype": "i32", "shape": shape, "kind": "workspace"}
            lists = [B(name + n) for n in (".work_p", ".count_p", ".work_d", ".count_d")]
            args = [B("cu_seqlens"), lists[0], lists[1], self.V("seqs"), {"expr": C.attn_plan_items(hq, hk)}, lists[2], lists[3]]
            self.plans[name] = lists, C.attn_plan_op(hq, hk, cfg.max_seqs, dim), args
        return self.plans[name][0]

    def row_plan(self) -> list[dict]:
        """The table row and reach of every token, for attention that takes a row per token."""
        if "rows" not in self.plans:
            c = self.rows_call("")
            self.plans["rows"] = [self.B("row_seq")], self.ops.pop(c["op"]), c["args"]
        return self.plans["rows"][0]

    def embed(self, next_norm: str, prefill: bool, scale: float = 1.0, conv: dict | None = None) -> dict:
        """Token rows, times `scale`, into the residual and the first sublayer's normed input, convolved where that reads it so (`conv`,
        from `input_conv`); the plans in the same call, so that both programs have as many calls to every layer."""
        cfg, B, d = self.cfg, self.B, self.cfg.width
        args = [B("token_ids"), self.same("embed", (cfg.vocab, d)), self.same(next_norm, (d,)), B("x"), B("xn"), self.err]
        first = [(o, more) for _, o, more in self.plans.values()] if prefill else []
        own = lambda: K.resid_embed_op(d, cfg.vocab, cfg.eps, self.act, scale)
        if conv and prefill:
            first.insert(0, (conv["op"](), conv["args"]))
        elif conv:
            args, own = args + conv["args"], lambda: K.resid_embed_op(d, cfg.vocab, cfg.eps, self.act, scale, conv["fused"])
        name = self.op("embed" + ("_p" if prefill else "_d"), lambda: K.chain_ops(own(), *[o for o, _ in first]))
        return {"op": name, "label": "embed", "args": args + [a for _, more in first for a in more]}

    # ---- a sublayer that reads its input plus a convolution of it ----
    def input_conv(self, tensor: str, taps: int, st: str, prefill: bool) -> dict:
        """xn -> `xc`, its last rows in lines `st`: in a decode call a part of the kernel that makes xn (`fused`: what its op takes,
        `args`: at the end), in a ragged one an op behind it."""
        cfg, d, A, B, V = self.cfg, self.cfg.width, self.act, self.B, self.V
        line = K.conv_line_bytes(d, taps, A)
        self.states[st] = {"bytes_per_seq": line}
        self.room("xc", d)
        tail = [self.same(tensor, (d, taps)), B("xc"), {"state": st}, B("lines")]
        return {"tag": f"{taps}x{line}", "fused": (taps, line), "op": lambda: K.conv_add_op(d, taps, line, A),
                "args": [B("xn"), *tail, B("cu_seqlens"), V("seqs"), V("tokens")] if prefill else tail}

    # ---- latent attention with a rotated part ----
    def latent(self, p: str, kv: str, m: dict, prefill: bool, tables: list[dict], *, x: str = "xn", halves: bool = True, sink: bool = False, gate: bool = False,
               window: int = C.I32_MAX) -> list[dict]:
        """Queries through a latent, one rotated key part for all heads, its rows in state `kv`: x -> y. `tables`: the rotation's;
        `sink`: a score per head in the denominator; `gate`: a sigmoid per head on the results; `window`: positions a row sees."""
        cfg, d, A, es, B, V, S, T = self.cfg, self.cfg.width, self.act, self.es, self.B, self.V, self.cfg.max_seqs, self.cfg.max_tokens
        z, sfx, page, W, err, eps = latent_sizes(m), "_p" if prefill else "_d", cfg.page_size, cfg.table_width, self.err, cfg.eps
        H, dim, rot, vdim, rank, qr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], z["rank"], m["q_rank"]
        self.states[kv] = {"bytes_per_token": z["down"] * es}
        w_in, down = self.rows_weight(f"w.{p}down", d, [(p + "dq", qr), (p + "dkv", z["down"])] + ([(p + "g", H)] if gate else []))
        # the unrotated rows of every head, then the rotated ones; filled up to whole 16-byte vectors of output
        head = lambda h, lo, hi: {"tensor": p + "uq", "rows": [h * (dim + rot) + lo, h * (dim + rot) + hi]}
        rows = z["q"] + z["rot"]
        qc = -(-rows // 8) * 8
        fill = [{"tensor": p + "uq", "rows": [0, 1]}] * (qc - rows)
        w_uq = self.weight(f"w.{p}uq", (qc, qr), *[head(h, 0, dim) for h in range(H)], *[head(h, dim, dim + rot) for h in range(H)], *fill)
        for name, cols in (("down", down), ("q_low", qr), ("q", qc), ("qlat", z["lat"]), ("olat", z["lat"]), ("attn", z["v"]), ("y", d)):
            self.room(name, cols)
        form = ("" if halves else "n") + ("" if window == C.I32_MAX else f"w{window}") + (f"g{down}" if gate else "")
        prep = self.op(f"latent_prep_{rank}x{rot}x{qr}x{down}" + ("" if halves else "n"), lambda: K.latent_prep_op(rank, rot, qr, down, qr, cfg.context, eps, A, halves))
        uk = self.same(p + "uk", (z["q"], rank))
        tiles, ukt = K.head_tiles(rank, dim, qc, z["lat"], A), f"ukt.{p.split('.')[0]}"
        if tiles and ukt not in self.bufs:      # the tensor-core form wants W_uk with a latent column per row: turned once, at load
            self.bufs[ukt] = {"dtype": "bf16", "shape": [H, rank, dim], "kind": "carry"}
            self.once.append({"op": self.op(f"transpose_{H}x{dim}x{rank}", lambda: K.transpose_heads_op(H, dim, rank)), "label": p + "ukt", "args": [uk, B(ukt)]})
        up = self.op(f"q_up_{H}x{dim}x{rank}x{qc}", lambda: K.head_linear_op(H, rank, dim, act=A, rows_max=T, lda=qc, ldc=z["lat"], transposed=not tiles))
        v_up = self.op(f"v_up_{H}x{vdim}x{rank}", lambda: K.head_linear_op(H, vdim, rank, act=A, rows_max=T, lda=z["lat"], ldc=z["v"]))
        attn = self.op(f"latent_attn{sfx}_{H}x{rank}x{rot}x{qc}{form}_{m['scale']!r}", lambda: K.latent_rot_attn_op(
            H, rank, rot, float(m["scale"]), page, W, cfg.context, qc, prefill, A, seqs_max=S, sink=sink, halves=halves, window=window, gate_stride=down if gate else 0))
        lens = [B("row_len"), err, *self.row_plan()] if prefill else [B("seq_lens"), err]
        extra = ([self.same(p + "sink", (H,))] if sink else []) + ([B("down", (qr + z["down"]) * es)] if gate else [])
        return [
            self.linear("lin", down, d, B(x), w_in, B("down"), label=p + "down"),
            {"op": prep, "label": p + "prep", "args": [B("down"), {"state": kv}, B("q_low"), B("positions"), B("slot_mapping"), *tables, self.same(p + "dkv.norm", (rank,)),
                                                       self.same(p + "dq.norm", (qr,)), err]},
            self.linear("lin", qc, qr, B("q_low"), w_uq, B("q"), label=p + "uq"),
            {"op": up, "label": p + "q_up", "args": [B("q"), B(ukt) if tiles else uk, B("qlat"), V("tokens"), err]},
            {"op": attn, "label": p + "attn", "args": [B("qlat"), {"state": kv}, B("olat"), B("block_table"), *lens, B("q", z["q"] * es), *tables, *extra]},
            {"op": v_up, "label": p + "v_up", "args": [B("olat"), self.same(p + "uv", (z["v"], rank)), B("attn"), V("tokens"), err]},
            self.linear("lin", d, z["v"], B("attn"), self.same(p + "o", (d, z["v"])), B("y"), label=p + "o"),
        ]

    # ---- linear attention with a decay per key channel ----
    def linear_attention(self, p: str, st: str, H: int, dk: int, dv: int, stride: int, ptrs, z, prefill: bool, norm, norm_shared: bool, u, q_scale, out, out_stride,
                         out_scale) -> list[dict]:
        """The recurrence from its projections (`ptrs`: q, k, v, gate) to the gated rows in `out`."""
        cfg, A, eps, B, V = self.cfg, self.act, self.cfg.eps, self.B, self.V
        sfx, fused = "_p" if prefill else "_d", not prefill and K.lin_fused(dv)
        tag = f"{sfx}_{H}x{dk}x{dv}x{stride}x{out_stride}" + ("u" if u else "") + f"_{out_scale!r}"

        def make():
            rule = K.lin_rule_op(H, dk, dv, stride, z["line"], z["s_off"], prefill, A, bonus=u is not None, q_scale=q_scale, fused=fused, norm_shared=norm_shared,
                                 out_stride=out_stride, out_scale=out_scale, eps=eps, rows_max=cfg.max_tokens, seqs_max=cfg.max_seqs)
            if fused:
                return rule
            ng = K.lin_norm_gate_op(H, dv, stride, norm_shared, out_stride, out_scale, eps, A)
            return K.chain_ops(rule, ng, inner={(0, 5 if u else 4): "o", (1, 0): "o"}, scratch={"o": {"dtype": "f32", "shape": ["tokens", H * dv]}})

        q, k, v, gate = ptrs
        head, cu = [q, k, v, B("alpha"), *([u] if u else [])], [B("cu_seqlens")] if prefill else []
        state = [{"state": st}, B("lines"), *cu]
        args = [*head, out, *state, gate, norm, V("seqs")] if fused else [*head, *state, V("seqs"), gate, norm, out]
        return [{"op": self.op(f"lin{tag}", make), "label": p + "rule", "args": args}]

    def gla(self, p: str, st: str, m: dict, rank: int, prefill: bool) -> list[dict]:
        """Gated linear attention of tensors `p`, its state in lines `st`, its decays through `rank` columns: xn -> y."""
        d, A, es, B = self.cfg.width, self.act, self.es, self.B
        z = gla_sizes(m)
        H, dk, dv, q, v = m["heads"], m["dim"], m["vdim"], z["q"], z["v"]
        self.states[st] = {"bytes_per_seq": z["line"]}
        w_in, proj = self.rows_weight(f"w.{p}qkvga", d, [(p + "q", q), (p + "k", q), (p + "v", v), (p + "g", v), (p + "a1", rank)])
        self.room("proj", proj); self.room("alpha", q, "f32"); self.room("mixed", v); self.room("y", d)
        decay = self.op(f"decay_{q}x{rank}x{proj}_{m['tau']!r}", lambda: K.decay_op(q, rank, proj, "root", m["tau"], A))
        col = lambda c: B("proj", c * es)
        return [
            self.linear("lin", proj, d, B("xn"), w_in, B("proj"), label=p + "in"),
            {"op": decay, "label": p + "decay", "args": [col(2 * q + 2 * v), self.same(p + "a2", (q, rank)), self.same(p + "a2.b", (q,)), B("alpha"), self.V("tokens")]},
            *self.linear_attention(p, st, H, dk, dv, proj, (col(0), col(q), col(2 * q), col(2 * q + v)), z, prefill, self.same(p + "norm", (dv,)), True, None,
                                   dk ** -0.5, B("mixed"), v, 1.0),
            self.linear("lin", d, v, B("mixed"), self.same(p + "o", (d, v)), B("y"), label=p + "o"),
        ]

    # ---- feed-forward ----
    def dense(self, p: str, ff: int, glu: str, bias: bool = False) -> list[dict]:
        """Gate and up projections with their gated unit, and the projection back: xn -> y. `bias`: gate and up have one each (the
        way back's is left to whoever adds y to the residual)."""
        d, B = self.cfg.width, self.B
        self.room("act", ff); self.room("y", d)
        base = ("glu" if glu == "swiglu" else glu) + ("_bias" if bias else "")
        b = self.weight(f"w.{p}mlp.gu.b", (2 * ff,), p + "mlp.gate.b", p + "mlp.up.b") if bias else None
        return [
            self.linear(base, 2 * ff, d, B("xn"), self.weight(f"w.{p}mlp.gu", (2 * ff, d), p + "mlp.gate", p + "mlp.up"), B("act"), label=p + "gate_up", bias=b, epilogue=glu),
            self.linear("lin", d, ff, B("act"), self.same(p + "mlp.down", (d, ff)), B("y"), label=p + "down"),
        ]

    def shared(self, p: str, ff: int) -> list[dict]:
        """An expert of every token: xn -> `shared.y`."""
        d, B = self.cfg.width, self.B
        self.room("shared.act", ff); self.room("shared.y", d)
        return [
            self.linear("glu", 2 * ff, d, B("xn"), self.weight(f"w.{p}mlp.shared.gu", (2 * ff, d), p + "mlp.shared.gate", p + "mlp.shared.up"), B("shared.act"),
                        label=p + "shared_gate_up", epilogue="swiglu"),
            self.linear("lin", d, ff, B("shared.act"), self.same(p + "mlp.shared.down", (d, ff)), B("shared.y"), label=p + "shared_down"),
        ]

    def routed(self, p: str, experts: int, top: int, ff: int, route, glu: str = "swiglu", limit: float = 0.0, router: tuple[dict, int] | None = None) -> list[dict]:
        """Routed experts up to their own rows: xn -> `moe.y` (expert-sorted), `moe.perm`, `moe.w`. `route(logits, ids, weights)` makes
        the call that picks them; an id from `experts` on has no row (`moe.perm` -1). `router`: a matrix of more rows than experts,
        and their number."""
        d, B = self.cfg.width, self.B
        w_router, outputs = router or (self.same(p + "mlp.router", (experts, d)), experts)
        self.room("moe.logits", outputs, "f32"); self.room("moe.ids", top, "i32"); self.room("moe.w", top, "f32")
        return [self.linear("router", outputs, d, B("xn"), w_router, B("moe.logits"), label=p + "router", epilogue="f32"), route(B("moe.logits"), B("moe.ids"), B("moe.w")),
                *self.experts(p, experts, top, ff, glu, limit)]

    def table_routed(self, p: str, experts: int, top: int, ff: int) -> list[dict]:
        """As `routed` with no router: tensor `<p>mlp.table` names the experts of every token id, all with one weight."""
        cfg, B = self.cfg, self.B
        self.room("moe.ids", top, "i32"); self.room("moe.w", top, "f32")
        op = self.op(f"moe_table_{experts}x{top}", lambda: K.route_table_op(experts, top, cfg.vocab))
        return [{"op": op, "label": p + "route", "args": [B("token_ids"), self.same(p + "mlp.table", (cfg.vocab, top), "i32"), B("moe.ids"), B("moe.w"), self.V("tokens"),
                                                          self.err]}, *self.experts(p, experts, top, ff)]

    def experts(self, p: str, experts: int, top: int, ff: int, glu: str = "swiglu", limit: float = 0.0) -> list[dict]:
        """The chosen experts (`moe.ids`) of every row."""
        cfg, d, B = self.cfg, self.cfg.width, self.B
        E, k, T, A, err = experts, top, cfg.max_tokens, self.act, self.err
        self.room("moe.perm", k, "i32")
        self.room("moe.x", k * d); self.room("moe.act", k * ff); self.room("moe.y", k * d)
        tiles = T * k // K.routed_tile_rows(A, d, ff) + E
        for name, shape in (("moe.offsets", [E + 1]), ("moe.tiles", [tiles, 4]), ("moe.tile_count", [1]), ("moe.rows", [1])):
            have = self.bufs.get(name, {"shape": [0]})["shape"]
            self.bufs[name] = {"dtype": "i32", "shape": [max(have[0], shape[0]), *shape[1:]], "kind": "workspace"}
        tag = f"{d}x{ff}x{E}x{k}" + (f"_{glu}{limit!r}" if glu != "swiglu" else "")
        if f"moe_plan_{tag}" not in self.ops:
            for n, o in K.routed_ops(d, ff, E, k, T, A, glu, limit).items():
                self.ops[f"{n}_{tag}"] = o
        n = {"expr": {"mul": ["tokens", k]}}
        w1 = self.weight(f"w.{p}mlp.w1", (E, 2 * ff, d), *[f"{p}mlp.e{e}.{t}" for e in range(E) for t in ("gate", "up")])
        w2 = self.weight(f"w.{p}mlp.w2", (E, d, ff), *[f"{p}mlp.e{e}.down" for e in range(E)])
        return [
            {"op": f"moe_plan_{tag}", "label": p + "plan", "args": [B("moe.ids"), B("moe.perm"), B("moe.offsets"), B("moe.tiles"), B("moe.tile_count"), B("moe.rows"), n, err]},
            {"op": f"moe_gather_{tag}", "label": p + "gather", "args": [B("xn"), B("moe.perm"), B("moe.x"), n]},
            {"op": f"moe_fc1_{tag}", "label": p + "fc1", "args": [B("moe.x"), w1, B("moe.act"), B("moe.tiles"), B("moe.tile_count"), n, err]},
            {"op": f"moe_fc2_{tag}", "label": p + "fc2", "args": [B("moe.act"), w2, B("moe.y"), B("moe.tiles"), B("moe.tile_count"), n, err]},
        ]

    # ---- from `hidden` to tokens ----
    def tail(self, head: str, prefill: bool) -> list[dict]:
        """Final norm, the projection by tensor `head`, and the next token of every sequence."""
        cfg, d, B = self.cfg, self.cfg.width, self.B
        pick = "last" if prefill else "each"
        norm = self.op("final_norm_" + pick, lambda: K.row_norm_op(d, cfg.eps, cfg.max_tokens, self.act, pick))
        calls = [{"op": norm, "label": "final_norm", "args": [B("hidden"), self.same("final.norm", (d,)), B("last_n"), *([B("cu_seqlens")] if prefill else [])]},
                 self.linear("head", cfg.vocab, d, B("last_n"), self.same(head, (cfg.vocab, d)), B("logits"), rows="seqs", label="lm_head", epilogue="f32")]
        if cfg.sampling:
            pick_op = self.op("sample", lambda: C.sample_op(cfg.vocab, "f32"))
            calls.append({"op": pick_op, "label": "sample", "args": [B("logits"), B("next_token"), *[B(n) for n in
                          ("temperature", "top_k", "top_p", "min_p", "seed", "seq_lens")]]})
        else:
            calls.append({"op": self.op("pick", lambda: C.argmax_op(cfg.vocab, "f32")), "label": "argmax", "args": [B("logits"), B("next_token")]})
        return calls

    def document(self, forward, head: str) -> dict:
        """The manifest; `forward(prefill)` writes the calls from the embedding to `hidden`."""
        cfg, d, B = self.cfg, self.cfg.width, self.B
        if cfg.sampling:
            self.bufs.setdefault("seq_lens", {"dtype": "i32", "shape": ["seqs"], "kind": "input", "fill": "seq_len"})
            for name, dt in (("temperature", "f32"), ("top_k", "i32"), ("top_p", "f32"), ("min_p", "f32"), ("seed", "i64")):
                self.bufs[name] = {"dtype": dt, "shape": ["seqs"], "kind": "input", "fill": name}
        prefill, decode = (forward(p) + self.tail(head, p) for p in (True, False))
        listed = self.op("final_norm_listed", lambda: K.row_norm_op(d, cfg.eps, cfg.max_tokens, self.act, "listed"))
        logits = [{"op": listed, "label": "want_norm", "args": [B("hidden"), B("w.final.norm"), B("want_n"), B("want_rows")]},
                  self.linear("head_rows", cfg.vocab, d, B("want_n"), B("w." + head), B("want_logits"), rows="wanted", label="want_head", epilogue="f32")]
        doc = {
            "schema_version": 7, "model": cfg.name,
            "vars": {"tokens": {"max": cfg.max_tokens, "axis": "rows"}, "seqs": {"max": cfg.max_seqs, "axis": "groups"}, "wanted": {"max": WANTED}},
            "states": self.states, "buffers": self.bufs, "modules": {}, "ops": self.ops,
            "programs": {
                "prefill": {"batch": {"groups": cfg.max_seqs, "rows": "tokens"}, "calls": prefill},
                "decode": {"batch": {"groups": cfg.max_seqs, "rows": 1}, "graph": True, "calls": decode},
                "logits": {"calls": logits},
            },
        }
        if self.once:
            doc["programs"]["load"] = {"once": True, "calls": self.once}
        used = {l["module"] for o in self.ops.values() for l in o["impl"]["launches"]}
        doc["modules"] = {n: m for n, m in C.modules_for(sorted(used)).items() if n in used}
        return doc


def gla_sizes(m: dict) -> dict:
    q, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
    line, s_off = K.lin_line_bytes(m["heads"], m["dim"], m["vdim"])
    return {"q": q, "v": v, "line": line, "s_off": s_off}


def latent_sizes(m: dict) -> dict:
    H, r = m["heads"], m["kv_rank"]
    return {"q": H * m["dim"], "rot": H * m["rot_dim"], "v": H * m["vdim"], "rank": r, "lat": H * r, "down": r + m["rot_dim"]}


# ---- checkpoints -------------------------------------------------------------------------------------------
def load_random(rt, shapes: dict, random, seed: int, std: float) -> None:
    """Fill the runtime's weights with a family's synthetic checkpoint, tensor by tensor on the runtime's device."""
    order = {n: i for i, n in enumerate(shapes)}

    def provider(name: str) -> torch.Tensor:
        dev = rt.tensor("x").device
        g = torch.Generator(device=dev).manual_seed(seed * 1000003 + order[name])
        return random(name, shapes[name], g, dev, std)

    rt.load_tensors(provider)


def save_folder(path, config: dict, weights: dict[str, torch.Tensor]) -> None:
    """A checkpoint folder: config.json and model.safetensors."""
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(config, indent=1))
    C.write_safetensors(path / "model.safetensors", weights)

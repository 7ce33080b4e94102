"""Barotar: a decoder whose layers are listed one by one. A layer's mixer is gated linear attention (a decay per key channel), or
two mixers side by side on one input: grouped-query attention in a sliding window (norms on q and k, rotary pairs of
neighbours, capped scores, a sink per head) and RWKV-style time mixing (token shift, a decay per key channel, a bonus for the
current token). Its feed-forward is a dense GEGLU, routed experts with a clamped gated unit chosen inside the best groups, or
none. Every sublayer is normed before and after, and the head is the embedding table.

Manifest generator, checkpoint names and synthetic weights. A layer with linear attention owns a per-sequence line (the previous
row when it shifts, then S in f32), one with attention a paged state of its keys and values. `dtype` "f32" is the exact form:
every activation, cached row and product in 32-bit over the same bf16 weights.

A program runs, per sublayer: mixer or feed-forward on the normed residual -> one kernel that norms the result, adds it and
makes the next sublayer's normed input. The two halves of a parallel mixer leave their rows, already scaled, side by side in one
buffer, and one product with both output projections, put next to each other when the weights are loaded, adds them up.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path

import torch

from . import blocks as K
from . import common as C
from . import listed
from .listed import Listed, gla_sizes, load_random


@dataclass
class BarotarConfig:
    name: str = "barotar"
    width: int = 2304
    vocab: int = 163840
    eps: float = 1e-6
    blocks: list = field(default_factory=list)     # the entries of config.json's `layers`
    ranks: list = field(default_factory=list)      # per layer: width of the decay's low-rank projection (a tensor's shape says it)
    layers: int | None = None                      # use only the first so many
    dtype: str = "bf16"                            # activations: bf16 | f32
    page_size: int = 64
    max_tokens: int = 8192
    max_seqs: int = 256
    max_context: int | None = None
    sampling: bool = False

    @property
    def depth(self) -> list:
        return self.blocks if self.layers is None else self.blocks[:self.layers]

    @property
    def context(self) -> int:
        return self.max_context or 8192

    @property
    def table_width(self) -> int:
        return -(-self.context // self.page_size)


_MIXER_KEYS = {"gla": {"dim", "heads", "tau", "vdim"}, "parallel": {"left", "left_scale", "right", "right_scale"}}
_LEFT_KEYS = {"dim", "heads", "kv_heads", "mask", "rot", "scale", "softcap", "vdim"}
MU = "rkvgw"          # the rows of a token shift, in the order they lie side by side


def low_rank(i: int, kind: str) -> str:
    """The tensor whose first extent is layer i's decay rank."""
    return f"l{i}.mix." + ("a1" if kind == "gla" else "right.w1")


def from_config(doc: dict, ranks: list[int], **over) -> BarotarConfig:
    """config.json and the decays' ranks -> the configuration; `over`: fields of the serving side (dtype, max_seqs, ..)."""
    for i, b in enumerate(doc["layers"]):
        if b["type"] not in _MIXER_KEYS:
            raise ValueError(f"layer {i}: unknown mixer `{b['type']}`; known: {', '.join(sorted(_MIXER_KEYS))}")
        m = b["mixer"]
        missing = _MIXER_KEYS[b["type"]] - set(m)
        if b["type"] == "parallel" and not missing:
            missing = (_LEFT_KEYS - set(m["left"])) | ({"dim", "heads"} - set(m["right"]))
        if missing:
            raise ValueError(f"layer {i}: mixer `{b['type']}` lacks {sorted(missing)}")
        if b["mlp"] is not None and b["mlp"]["kind"] not in ("dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward `{b['mlp']['kind']}`")
    return BarotarConfig(name=over.pop("name", "barotar"), width=doc["width"], vocab=doc["vocab"], eps=doc["norm"]["eps"], blocks=doc["layers"],
                         ranks=list(ranks), **over)


def from_folder(path, **over) -> BarotarConfig:
    doc = json.loads((Path(path) / "config.json").read_text())
    shapes = {}
    for f in sorted(Path(path).glob("*.safetensors")):
        shapes |= C.safetensors_shapes(f)
    return from_config(doc, [shapes[low_rank(i, b["type"])][0] for i, b in enumerate(doc["layers"])], **over)


def to_config(cfg: BarotarConfig) -> dict:
    """The config.json of a configuration."""
    return {"architecture": "Barotar", "layers": cfg.depth, "norm": {"eps": cfg.eps}, "vocab": cfg.vocab, "width": cfg.width}


def _gla(heads, dim, vdim, tau):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def _parallel(heads, kv_heads, dim, vdim, window, rot, base, scale, cap, right_heads, right_dim, left_scale, right_scale):
    return "parallel", {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": {"base": base, "dims": rot},
                                 "scale": scale, "softcap": cap},
                        "right": {"heads": right_heads, "dim": right_dim}, "left_scale": left_scale, "right_scale": right_scale}


def _block(mixer, mlp) -> dict:
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def _dense(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def _moe(experts: int, top: int, ff: int, groups: int, keep: int, limit: float) -> dict:
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


TINY_BAROTAR = BarotarConfig(
    name="tiny-barotar", width=128, vocab=256, page_size=16, max_tokens=256, max_seqs=8, max_context=512,
    blocks=[_block(_parallel(4, 2, 64, 64, 40, 32, 1e4, 0.125, 20.0, 3, 32, 0.7, 0.9), _moe(12, 2, 40, 3, 2, 3.0)),
            _block(_gla(3, 24, 40, 8.0), _dense(160)),
            _block(_parallel(6, 3, 32, 48, 70, 16, 1e5, 0.2, 25.0, 2, 48, 1.2, 0.5), None)], ranks=[8, 16, 24])
# the width, depth, vocabulary and experts of the 48B-A3B shape class; every fourth layer gated linear attention
BAROTAR_LARGE = BarotarConfig(
    name="barotar-48b-a3b", width=2304, vocab=163840,
    blocks=[_block(_gla(16, 128, 256, 16.0) if i % 4 == 3 else _parallel(32, 4, 128, 128, 1024, 64, 1e6, 128 ** -0.5, 30.0, 32, 64, 0.8, 0.9),
                   _moe(256, 8, 1024, 8, 4, 7.0)) for i in range(27)], ranks=[64] * 27)


# ---- sizes of a layer ---------------------------------------------------------------------------------------
def parallel_sizes(m: dict, width: int) -> dict:
    l, r = m["left"], m["right"]
    inner = r["heads"] * r["dim"]
    line, s_off = K.lin_line_bytes(r["heads"], r["dim"], r["dim"], width)
    return {"q": l["heads"] * l["dim"], "k": l["kv_heads"] * l["dim"], "v": l["kv_heads"] * l["vdim"], "o": l["heads"] * l["vdim"], "inner": inner,
            "token": l["kv_heads"] * (l["dim"] + l["vdim"]), "line": line, "s_off": s_off}


def weight_names(cfg: BarotarConfig) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor name -> shape; every tensor is bf16."""
    d = cfg.width
    out = {"embed": (cfg.vocab, d)}
    for i, b in enumerate(cfg.depth):
        p, m, f, rank = f"l{i}.", b["mixer"], b["mlp"], cfg.ranks[i]
        for n in ("1",) + (("2",) if f is not None else ()):
            out |= {f"{p}norm{n}": (d,), f"{p}norm{n}b": (d,)}
        if b["type"] == "gla":
            z, q = gla_sizes(m), p + "mix."
            out |= {q + "q": (z["q"], d), q + "k": (z["q"], d), q + "v": (z["v"], d), q + "g": (z["v"], d), q + "o": (d, z["v"]), q + "norm": (m["vdim"],),
                    q + "a1": (rank, d), q + "a2": (z["q"], rank), q + "a2.b": (z["q"],)}
        else:
            z, l, r = parallel_sizes(m, d), p + "mix.left.", p + "mix.right."
            n = z["inner"]
            out |= {l + "q": (z["q"], d), l + "k": (z["k"], d), l + "v": (z["v"], d), l + "q.norm": (m["left"]["dim"],), l + "k.norm": (m["left"]["dim"],),
                    l + "sink": (m["left"]["heads"],), l + "o": (d, z["o"])}
            out |= {f"{r}mu.{s}": (d,) for s in MU} | {r + s: (n, d) for s in "rkvg"}
            out |= {r + "w1": (rank, d), r + "w2": (n, rank), r + "w0": (n,), r + "u": (m["right"]["heads"], m["right"]["dim"]), r + "norm": (n,), r + "o": (d, n)}
        if f is not None and f["kind"] == "dense":
            out |= {p + "mlp.gate": (f["ff"], d), p + "mlp.up": (f["ff"], d), p + "mlp.down": (d, f["ff"])}
        elif f is not None:
            for e in range(f["router"]["experts"]):
                q, ff = f"{p}mlp.e{e}.", f["expert"]["ff"]
                out |= {q + "gate": (ff, d), q + "up": (ff, d), q + "down": (d, ff)}
            out[p + "mlp.router"] = (f["router"]["experts"], d)
    out["final.norm"] = (d,)
    return out


def _random(name: str, shape, g, device, std: float) -> torch.Tensor:
    n = lambda: torch.randn(shape, generator=g, device=device)
    last = name.rsplit(".", 1)[-1]
    if "norm" in last:
        t = 1 + 0.1 * n()
    elif ".mu." in name:
        t = torch.rand(shape, generator=g, device=device)
    elif last == "w0":
        t = -3 + 1.5 * n()                      # decays from a few tokens to hundreds
    elif last == "b":
        t = 2 + n()
    elif last == "u":
        t = 0.5 + 0.5 * n()
    elif last == "sink":
        t = n()
    elif last == "router":
        t = 10 * std * n()                      # a router with opinions
    elif name == "embed":
        t = n()
    else:
        t = std * n()
    return t.to(torch.bfloat16)


def random_weights(cfg: BarotarConfig, seed: int = 0, device: str = "cpu", std: float = 0.02) -> dict[str, torch.Tensor]:
    g = torch.Generator(device=device).manual_seed(seed)
    return {n: _random(n, s, g, device, std) for n, s in weight_names(cfg).items()}


def load_random_weights(rt, cfg: BarotarConfig, seed: int = 0, std: float = 0.02) -> None:
    load_random(rt, weight_names(cfg), _random, seed, std)


def save_folder(path, cfg: BarotarConfig, weights: dict[str, torch.Tensor]) -> None:
    listed.save_folder(path, to_config(cfg), weights)


# ---- the manifest -------------------------------------------------------------------------------------------
def build_manifest(cfg: BarotarConfig) -> dict:
    d, A, S, W, page, eps = cfg.width, cfg.dtype, cfg.max_seqs, cfg.table_width, cfg.page_size, cfg.eps
    m_ = Listed(cfg)
    layers, es, bufs, states, err = cfg.depth, m_.es, m_.bufs, m_.states, m_.err
    B, V, op, room, weight, same, linear = m_.B, m_.V, m_.op, m_.room, m_.weight, m_.same, m_.linear
    windows = [i for i, b in enumerate(layers) if b["type"] == "parallel"]
    tiled = {i: K.window_tiles(*(layers[i]["mixer"]["left"][k] for k in ("heads", "kv_heads", "dim", "vdim")), page, A) for i in windows}
    untiled = [i for i in windows if not tiled[i]]
    m_.inputs(f"kv.l{windows[0]}" if windows else None, "lin.l0", positions=bool(windows), row_plan=bool(untiled))
    room("x", d, "f32")
    room("xn", d)
    m_.outputs()

    # every sublayer in order: its norm before, its norm after
    subs = [(f"l{i}.norm{q}", f"l{i}.norm{q}b") for i, b in enumerate(layers) for q in ((1, 2) if b["mlp"] is not None else (1,))]

    def finish(at: int, y, label: str, routed: int = 0, extra=()) -> dict:
        """Sublayer `at`'s normed result onto the residual; the next one's input, or the residual itself after the last."""
        post = same(subs[at][1], (d,))
        if at + 1 == len(subs):
            name = op(f"resid_last_{routed}", lambda: K.resid_mix_op(d, eps, A, routed, last=True))
            return {"op": name, "label": label, "args": [B("x"), y, post, B("hidden"), *extra]}
        name = op(f"resid_mix_{routed}", lambda: K.resid_mix_op(d, eps, A, routed))
        return {"op": name, "label": label, "args": [B("x"), y, post, same(subs[at + 1][0], (d,)), B("xn"), *extra]}

    def gla(i: int, at: int, prefill: bool) -> list[dict]:
        p = f"l{i}.mix."
        return m_.gla(p, f"lin.l{i}", layers[i]["mixer"], cfg.ranks[i], prefill) + [finish(at, B("y"), p + "out")]

    def parallel(i: int, at: int, prefill: bool) -> list[dict]:
        m, p, rank = layers[i]["mixer"], f"l{i}.mix.", cfg.ranks[i]
        z, l, r, lp, rp = parallel_sizes(m, d), m["left"], m["right"], f"l{i}.mix.left.", f"l{i}.mix.right."
        hq, hk, dim, vdim, H, dk, n = l["heads"], l["kv_heads"], l["dim"], l["vdim"], r["heads"], r["dim"], z["inner"]
        kv, st, both, sfx = f"kv.l{i}", f"lin.l{i}", z["o"] + n, "_p" if prefill else "_d"
        states[kv], states[st] = {"bytes_per_token": z["token"] * es}, {"bytes_per_seq": z["line"]}
        w_in, qkv = m_.rows_weight(f"w.{lp}qkv", d, [(lp + "q", z["q"]), (lp + "k", z["k"]), (lp + "v", z["v"])])
        room("qkv", qkv); room("shifted", len(MU) * d); room("rkvg", 4 * n); room("low", rank, "f32"); room("alpha", n, "f32"); room("mixed", both); room("y", d)
        # left: window attention into columns 0 .. o of `mixed`
        cos_sin = m_.rotary(l["rot"]["dims"], l["rot"]["base"])
        prep = op(f"prep_{hq}x{hk}x{dim}x{vdim}x{l['rot']['dims']}", lambda: K.qk_prep_op(hq, hk, dim, vdim, l["rot"]["dims"], page, qkv, cfg.context, eps, A))
        attn = op(f"window_attn{sfx}_{hq}x{hk}x{dim}x{vdim}x{l['mask']['size']}x{both}_{l['scale']!r}_{l['softcap']!r}_{m['left_scale']!r}", lambda: K.window_attn_op(
            hq, hk, dim, vdim, l["mask"]["size"], l["scale"], l["softcap"], page, W, qkv, both, m["left_scale"], prefill, A, seqs_max=S))
        lens, lists = B("seq_lens"), []
        if prefill and tiled[i]:
            lists = [B("cu_seqlens"), *m_.lists_of(hq, hk, dim)]
        elif prefill:
            lens, lists = B("row_len"), m_.row_plan()
        calls = [
            linear("lin", qkv, d, B("xn"), w_in, B("qkv"), label=lp + "qkv"),
            {"op": prep, "label": lp + "prep", "args": [B("qkv"), {"state": kv}, B("positions"), B("slot_mapping"), *cos_sin, same(lp + "q.norm", (dim,)),
                                                        same(lp + "k.norm", (dim,)), err]},
            {"op": attn, "label": lp + "attn", "args": [B("qkv"), {"state": kv}, B("mixed"), B("block_table"), lens, same(lp + "sink", (hq,)), err, *lists]},
        ]
        # right: token shift, projections of the five mixes, the recurrence into columns o .. of `mixed`
        mu = weight(f"w.{rp}mu", (len(MU), d), *[f"{rp}mu.{s}" for s in MU])
        shift = op(f"shift{sfx}_{z['line']}", lambda: K.token_shift_op(d, len(MU), z["line"], prefill, A))
        heads = op(f"rkvg_{n}x{d}", lambda: K.head_linear_op(4, n, d, act=A, rows_max=cfg.max_tokens, lda=len(MU) * d, ldc=4 * n))
        decay = op(f"decay_{n}x{rank}", lambda: K.decay_op(n, rank, rank, "double_exp"))
        col = lambda c: B("rkvg", c * n * es)
        cu = [B("cu_seqlens")] if prefill else []
        calls += [
            {"op": shift, "label": rp + "shift", "args": [B("xn"), mu, B("shifted"), {"state": st}, B("lines"), *cu, V("seqs")]},
            {"op": heads, "label": rp + "rkvg", "args": [B("shifted"), weight(f"w.{rp}rkvg", (4, n, d), *[rp + s for s in "rkvg"]), B("rkvg"), V("tokens"), err]},
            linear("low", rank, d, B("shifted", 4 * d * es), same(rp + "w1", (rank, d)), B("low"), label=rp + "w1", epilogue="f32", lda=len(MU) * d),
            {"op": decay, "label": rp + "decay", "args": [B("low"), same(rp + "w2", (n, rank)), same(rp + "w0", (n,)), B("alpha"), V("tokens")]},
            *m_.linear_attention(rp, st, H, dk, dk, 4 * n, [col(c) for c in range(4)], z, prefill, same(rp + "norm", (n,)), False, same(rp + "u", (H, dk)), 1.0,
                              B("mixed", z["o"] * es), both, m["right_scale"]),
        ]
        # both output projections next to each other, so one product adds the halves up
        if f"o.l{i}" not in bufs:
            bufs[f"o.l{i}"] = {"dtype": "bf16", "shape": [d, both], "kind": "carry"}
            for part, cols, off in ((lp, z["o"], 0), (rp, n, z["o"])):
                name = op(f"copy_cols_{cols}of{both}", lambda: K.copy_cols_op(d, cols, both))
                m_.once.append({"op": name, "label": part + "o", "args": [same(part + "o", (d, cols)), B(f"o.l{i}", off * 2)]})
        return calls + [linear("lin", d, both, B("mixed"), B(f"o.l{i}"), B("y"), label=p + "o"), finish(at, B("y"), p + "out")]

    def dense(i: int, at: int) -> list[dict]:
        p = f"l{i}."
        return m_.dense(p, layers[i]["mlp"]["ff"], "geglu") + [finish(at, B("y"), p + "mlp.out")]

    def routed(i: int, at: int) -> list[dict]:
        f, p = layers[i]["mlp"], f"l{i}."
        r, x = f["router"], f["expert"]
        E, k, count, keep = r["experts"], r["top"], r["groups"]["count"], r["groups"]["keep"]
        route = op(f"moe_route_{E}x{k}_{keep}of{count}", lambda: K.route_groups_op(E, k, count, keep))
        pick = lambda logits, ids, w: {"op": route, "label": p + "route", "args": [logits, ids, w, V("tokens")]}
        return m_.routed(p, E, k, x["ff"], pick, "clamped", x["limit"]) + [finish(at, B("moe.y"), p + "mlp.out", k, [B("moe.perm"), B("moe.w")])]

    def forward(prefill: bool) -> list[dict]:
        calls, at = [], 0
        for i, b in enumerate(layers):
            calls += (gla if b["type"] == "gla" else parallel)(i, at, prefill)
            at += 1
            if b["mlp"] is not None:
                calls += (dense if b["mlp"]["kind"] == "dense" else routed)(i, at)
                at += 1
        return [m_.embed(subs[0][0], prefill), *calls]

    return m_.document(forward, "embed")

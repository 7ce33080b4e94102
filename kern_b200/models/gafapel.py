"""Gafapel: a decoder whose layers are listed one by one, each with its own mixer (Mamba-2, or latent attention without
positions behind an output gate) and feed-forward (dense SwiGLU, routed experts, or none); learned positions are added to
the token embedding and normed, and the residual is a set of hyper-connected streams kept in f32.

Manifest generator, checkpoint names and synthetic weights. A Mamba-2 layer owns a per-sequence state (convolution window
+ recurrent matrix), a latent layer a paged state of `kv_rank` columns per token. `dtype` "f32" is the exact form: every
activation, cached row and product in 32-bit over the same bf16 weights.

A program runs, per sublayer: mixer or feed-forward on the normed stream sum -> one kernel that puts the result into the
streams and makes the next sublayer's normed input. The last sublayer leaves the sum of the streams in `hidden` (a carry:
the rows of the last call), from which `prefill` / `decode` norm and project each sequence's last row and the `logits`
program any listed rows.
"""
from __future__ import annotations

import json
import re
from dataclasses import dataclass, field
from pathlib import Path

import torch

from . import blocks as K
from . import common as C


@dataclass
class GafapelConfig:
    name: str = "gafapel"
    width: int = 2304
    vocab: int = 163840
    streams: int = 4
    max_positions: int = 8192
    eps: float = 1e-6
    blocks: list = field(default_factory=list)     # the entries of config.json's `layers`
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
        return min(self.max_context or self.max_positions, self.max_positions)

    @property
    def table_width(self) -> int:
        return -(-self.context // self.page_size)


KINDS = ("mamba2", "latent_attention")
_MIXER_KEYS = {"mamba2": {"conv", "groups", "heads", "norm_groups", "state", "vdim"},
               "latent_attention": {"dim", "heads", "kv_rank", "scale", "vdim"}}


def kind_of(block: dict) -> str:
    """The mechanism of a layer type: `mamba2`, `mamba2_2`, ... are differently sized mixers of one kind."""
    m = re.fullmatch(r"(mamba2|latent_attention)(_\d+)?", block["type"])
    if not m:
        raise ValueError(f"unknown mixer `{block['type']}`; known: {', '.join(KINDS)}")
    return m.group(1)


def from_config(doc: dict, **over) -> GafapelConfig:
    """config.json -> the configuration; `over`: fields of the serving side (dtype, max_seqs, ..)."""
    for i, b in enumerate(doc["layers"]):
        missing = _MIXER_KEYS[kind_of(b)] - set(b["mixer"])
        if missing:
            raise ValueError(f"layer {i}: mixer `{b['type']}` lacks {sorted(missing)}")
        if b["mlp"] is not None and b["mlp"]["kind"] not in ("dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward `{b['mlp']['kind']}`")
    return GafapelConfig(name=over.pop("name", "gafapel"), width=doc["width"], vocab=doc["vocab"], streams=doc["streams"],
                         max_positions=doc["max_positions"], eps=doc["norm"]["eps"], blocks=doc["layers"], **over)


def from_folder(path, **over) -> GafapelConfig:
    return from_config(json.loads((Path(path) / "config.json").read_text()), **over)


def to_config(cfg: GafapelConfig) -> dict:
    """The config.json of a configuration."""
    return {"architecture": "Gafapel", "layers": cfg.depth, "max_positions": cfg.max_positions, "norm": {"eps": cfg.eps},
            "streams": cfg.streams, "vocab": cfg.vocab, "width": cfg.width}


def _mamba(heads, vdim, state, groups, conv, norm_groups, kind="mamba2"):
    return kind, {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _latent(heads, dim, vdim, kv_rank, scale):
    return "latent_attention", {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}


def _block(mixer, mlp) -> dict:
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def _dense(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def _moe(experts: int, top: int, ff: int) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


TINY_GAFAPEL = GafapelConfig(
    name="tiny-gafapel", width=128, vocab=256, streams=2, max_positions=512, page_size=16, max_tokens=256, max_seqs=8,
    blocks=[_block(_mamba(4, 32, 32, 2, 4, 4), _moe(8, 3, 40)), _block(_latent(4, 32, 48, 80, 0.2), _dense(160)),
            _block(_mamba(6, 16, 16, 1, 2, 1, "mamba2_2"), None), _block(_latent(4, 32, 48, 80, 0.2), _moe(8, 3, 40))])
# the shape class of the 48B latent-attention hybrid: every fourth layer latent attention, 256 experts of 1024, 8 per token
GAFAPEL_LARGE = GafapelConfig(
    name="gafapel-48b-a3b", width=2304, vocab=163840, streams=4, max_positions=8192,
    blocks=[_block(_latent(32, 128, 128, 512, 128 ** -0.5) if i % 4 == 3 else _mamba(64, 64, 128, 8, 4, 8), _moe(256, 8, 1024))
            for i in range(27)])


# ---- sizes of a layer ---------------------------------------------------------------------------------------
def mamba_sizes(m: dict, dtype: str) -> dict:
    inner = m["heads"] * m["vdim"]
    channels = inner + 2 * m["groups"] * m["state"]
    rows = inner + channels + m["heads"]
    line, s_off = K.ssd_line_bytes(m["heads"], m["vdim"], m["state"], channels, m["conv"], dtype)
    # the projection's rows are filled up to whole 16-byte vectors with copies of its first ones, which nobody reads
    return {"inner": inner, "channels": channels, "rows": rows, "proj": -(-rows // 8) * 8, "line": line, "s_off": s_off}


def latent_sizes(m: dict) -> dict:
    q, g, r = m["heads"] * m["dim"], m["heads"] * m["vdim"], m["kv_rank"]
    return {"q": q, "v": g, "rank": r, "lat": m["heads"] * r, "rows": q + g + r, "proj": -(-(q + g + r) // 8) * 8}


def weight_names(cfg: GafapelConfig) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor name -> shape; every tensor is bf16."""
    d, s = cfg.width, cfg.streams
    out = {"embed": (cfg.vocab, d), "pos": (cfg.max_positions, d), "embed.norm": (d,)}
    for i, b in enumerate(cfg.depth):
        p, m, f = f"l{i}.", b["mixer"], b["mlp"]
        out[p + "norm1"] = (d,)
        if f is not None:
            out[p + "norm2"] = (d,)
        if kind_of(b) == "mamba2":
            z = mamba_sizes(m, cfg.dtype)
            out |= {p + "mix.in": (z["rows"], d), p + "mix.conv": (z["channels"], m["conv"]), p + "mix.conv.b": (z["channels"],),
                    p + "mix.dt_bias": (m["heads"],), p + "mix.A_log": (m["heads"],), p + "mix.D": (m["heads"],),
                    p + "mix.norm": (z["inner"],), p + "mix.o": (d, z["inner"])}
        else:
            z = latent_sizes(m)
            out |= {p + "mix.q": (z["q"], d), p + "mix.dkv": (z["rank"], d), p + "mix.dkv.norm": (z["rank"],),
                    p + "mix.uk": (z["q"], z["rank"]), p + "mix.uv": (z["v"], z["rank"]), p + "mix.g": (z["v"], d),
                    p + "mix.o": (d, z["v"])}
        if f is not None and f["kind"] == "dense":
            out |= {p + "mlp.gate": (f["ff"], d), p + "mlp.up": (f["ff"], d), p + "mlp.down": (d, f["ff"])}
        elif f is not None:
            for e in range(f["router"]["experts"]):
                q, ff = f"{p}mlp.e{e}.", f["expert"]["ff"]
                out |= {q + "gate": (ff, d), q + "up": (ff, d), q + "down": (d, ff)}
            out |= {p + "mlp.router": (f["router"]["experts"], d), p + "mlp.router.b": (f["router"]["experts"],)}
        for q in ("hc1",) + (("hc2",) if f is not None else ()):
            out |= {f"{p}{q}.in": (s,), f"{p}{q}.out": (s,), f"{p}{q}.mix": (s, s)}
    out |= {"final.norm": (d,), "head": (cfg.vocab, d)}
    return out


def _random(name: str, shape, g, device, std: float) -> torch.Tensor:
    n = lambda: torch.randn(shape, generator=g, device=device)
    last = name.rsplit(".", 1)[-1]
    if "norm" in last:
        t = 1 + 0.1 * n()
    elif last == "A_log":
        t = torch.log(torch.empty(shape, device=device).uniform_(1.0, 8.0, generator=g))
    elif last == "dt_bias":
        t = -3 + n()
    elif last == "D":
        t = 1 + 0.1 * n()
    elif name.endswith(".conv"):
        t = 0.4 * n()
    elif name.endswith((".conv.b", ".router.b")):
        t = 0.1 * n()
    elif ".hc" in name:
        t = {"in": lambda: 1.0 / shape[0] + 0.1 * n(), "out": lambda: 1 + 0.1 * n(),
             "mix": lambda: torch.eye(shape[0], device=device) + 0.1 * n()}[last]()
    elif last == "router":
        t = 10 * std * n()                      # a router with opinions
    elif name in ("embed", "pos"):
        t = n()
    else:
        t = std * n()
    return t.to(torch.bfloat16)


def random_weights(cfg: GafapelConfig, seed: int = 0, device: str = "cpu", std: float = 0.02) -> dict[str, torch.Tensor]:
    g = torch.Generator(device=device).manual_seed(seed)
    return {n: _random(n, s, g, device, std) for n, s in weight_names(cfg).items()}


def load_random_weights(rt, cfg: GafapelConfig, seed: int = 0, std: float = 0.02) -> None:
    """Fill the runtime's weights with the synthetic checkpoint, tensor by tensor on the runtime's device."""
    shapes = weight_names(cfg)
    order = {n: i for i, n in enumerate(shapes)}

    def provider(name: str) -> torch.Tensor:
        dev = rt.tensor("x").device
        g = torch.Generator(device=dev).manual_seed(seed * 1000003 + order[name])
        return _random(name, shapes[name], g, dev, std)

    rt.load_tensors(provider)


def save_folder(path, cfg: GafapelConfig, weights: dict[str, torch.Tensor]) -> None:
    """A checkpoint folder: config.json and model.safetensors."""
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(to_config(cfg), indent=1))
    C.write_safetensors(path / "model.safetensors", weights)


# ---- the manifest -------------------------------------------------------------------------------------------
WANTED = 512          # most rows one call of the `logits` program projects


def build_manifest(cfg: GafapelConfig) -> dict:
    d, A, T, S, W = cfg.width, cfg.dtype, cfg.max_tokens, cfg.max_seqs, cfg.table_width
    if A not in K.ACT_BYTES:
        raise ValueError(f"dtype `{A}`: bf16 or f32")
    es, layers = K.ACT_BYTES[A], cfg.depth
    if not layers:
        raise ValueError("a model without layers")
    bufs, ops, states, once = {}, {}, {}, []
    B = lambda n, off=0: ({"buf": n, "offset": off} if off else {"buf": n})
    V = lambda n: {"var": n}
    err = B("error")

    def op(name: str, make) -> str:
        """An op under a name that says its sizes, made once."""
        if name not in ops:
            ops[name] = make()
        return name

    def room(name: str, cols: int, dtype: str = A, kind: str = "workspace") -> None:
        """A per-token buffer as wide as the widest layer that uses it."""
        have = bufs.get(name, {"shape": ["tokens", 0]})["shape"][1]
        bufs[name] = {"dtype": dtype, "shape": ["tokens", max(have, cols)], "kind": kind}

    def weight(name: str, shape, *tensors) -> dict:
        if name not in bufs:
            bufs[name] = {"dtype": "bf16", "shape": list(shape), "kind": "weight",
                          "bind": [t if isinstance(t, dict) else {"tensor": t} for t in tensors]}
        return B(name)

    def same(name: str, shape) -> dict:
        return weight("w." + name, shape, name)

    def linear(base: str, n: int, k: int, a, w, c, rows: str = "tokens", label: str = "", **kw) -> dict:
        name = op(f"{base}_{n}x{k}", lambda: K.linear_op(n, k, act=A, rows_var=rows, rows_max=T if rows == "tokens" else
                                                         (S if rows == "seqs" else WANTED), **kw))
        return {"op": name, "label": label, "args": [a, w, c, V(rows), err]}

    kinds = [kind_of(b) for b in layers]
    latents = [i for i, k in enumerate(kinds) if k == "latent_attention"]
    mambas = [i for i, k in enumerate(kinds) if k == "mamba2"]
    inp = lambda dt, shape, **kw: {"dtype": dt, "shape": shape, "kind": "input", **kw}
    bufs["token_ids"] = inp("i64", ["tokens"], fill="token", domain={"min": 0, "max": cfg.vocab - 1})
    bufs["positions"] = inp("i64", ["tokens"], fill="position", domain={"min": 0, "max": cfg.context - 1})
    bufs["cu_seqlens"] = inp("i32", [S + 1], fill="cu_seqlens")
    if latents:
        kv0 = f"kv.l{latents[0]}"
        bufs["slot_mapping"] = inp("i64", ["tokens"], fill="slot", domain={"index_into": kv0})
        bufs["seq_lens"] = inp("i32", ["seqs"], fill="seq_len")
        bufs["block_table"] = inp("i32", ["seqs", W], domain={"index_into": kv0, "stride": cfg.page_size})
        bufs["row_seq"] = {"dtype": "i32", "shape": ["tokens"], "kind": "workspace"}
        bufs["row_len"] = {"dtype": "i32", "shape": ["tokens"], "kind": "workspace"}
    if mambas:
        bufs["lines"] = inp("i32", [1, "seqs"], domain={"index_into": f"ssd.l{mambas[0]}"})
    bufs["next_token"] = {"dtype": "i64", "shape": ["seqs"], "kind": "output", "fill": "tokens"}
    bufs["error"] = {"dtype": "i32", "shape": [1], "kind": "output", "fill": "error"}
    room("x", cfg.streams * d, "f32")
    room("xn", d)
    room("hidden", d, "f32", "carry")
    bufs["last_n"] = {"dtype": A, "shape": ["seqs", d], "kind": "workspace"}
    bufs["logits"] = {"dtype": "f32", "shape": ["seqs", cfg.vocab], "kind": "workspace"}
    bufs["want_rows"] = inp("i32", ["wanted"])
    bufs["want_n"] = {"dtype": A, "shape": ["wanted", d], "kind": "workspace"}
    bufs["want_logits"] = {"dtype": "f32", "shape": ["wanted", cfg.vocab], "kind": "output"}

    # every sublayer in order: (its stream weights, its norm)
    subs = [(f"l{i}.hc{q}", f"l{i}.norm{q}") for i, b in enumerate(layers) for q in ((1, 2) if b["mlp"] is not None else (1,))]
    s = cfg.streams

    def finish(at: int, y, label: str, routed: int = 0, extra=()) -> dict:
        """Sublayer `at`'s result into the streams; the next one's input, or the sum of the streams after the last."""
        hc = subs[at][0]
        mix, out = same(hc + ".mix", (s, s)), same(hc + ".out", (s,))
        if at + 1 == len(subs):
            name = op(f"hyper_last_{routed}", lambda: K.hyper_last_op(d, s, A, routed))
            return {"op": name, "label": label, "args": [B("x"), y, mix, out, B("hidden"), *extra]}
        name = op(f"hyper_mix_{routed}", lambda: K.hyper_mix_op(d, s, cfg.eps, A, routed))
        nxt_hc, nxt_norm = subs[at + 1]
        return {"op": name, "label": label, "args": [B("x"), y, mix, out, same(nxt_hc + ".in", (s,)), same(nxt_norm, (d,)), B("xn"), *extra]}

    def mamba(i: int, at: int, prefill: bool) -> list[dict]:
        m, p, sfx = layers[i]["mixer"], f"l{i}.", "_p" if prefill else "_d"
        z = mamba_sizes(m, A)
        H, inner, ch, proj = m["heads"], z["inner"], z["channels"], z["proj"]
        st = f"ssd.l{i}"
        states[st] = {"bytes_per_seq": z["line"]}
        room("proj", proj); room("xbc", ch); room("ssd_y", inner, "f32"); room("ssd_n", inner); room("y", d)
        w_in = weight(f"w.{p}mix.in", (proj, d), p + "mix.in",
                      *([{"tensor": p + "mix.in", "rows": [0, proj - z["rows"]]}] if proj > z["rows"] else []))
        tag = f"{H}x{m['vdim']}x{m['state']}x{m['groups']}x{m['conv']}"
        cu = [B("cu_seqlens")] if prefill else []
        conv = op(f"conv{sfx}_{tag}", lambda: K.short_conv_op(ch, m["conv"], proj, z["line"], prefill, A, x_off=inner))
        rule = op(f"ssd{sfx}_{tag}", lambda: K.ssd_rule_op(H, m["vdim"], m["state"], m["groups"], proj, z["line"], z["s_off"], prefill, A))
        norm = op(f"ssd_norm_{inner}x{m['norm_groups']}x{proj}", lambda: K.ssd_gate_norm_op(inner, m["norm_groups"], proj, cfg.eps, A))
        return [
            linear("lin", proj, d, B("xn"), w_in, B("proj"), label=p + "in"),
            {"op": conv, "label": p + "conv", "args": [B("proj", inner * es), B("xbc"), {"state": st}, B("lines"), *cu,
                                                       same(p + "mix.conv", (ch, m["conv"])), same(p + "mix.conv.b", (ch,)), V("seqs"), V("tokens")]},
            {"op": rule, "label": p + "rule", "args": [B("xbc"), B("proj", (inner + ch) * es), B("ssd_y"), {"state": st}, B("lines"), *cu,
                                                       same(p + "mix.A_log", (H,)), same(p + "mix.dt_bias", (H,)), same(p + "mix.D", (H,)), V("seqs")]},
            {"op": norm, "label": p + "gnorm", "args": [B("ssd_y"), B("proj"), same(p + "mix.norm", (inner,)), B("ssd_n")]},
            linear("lin", d, inner, B("ssd_n"), same(p + "mix.o", (d, inner)), B("y"), label=p + "o"),
            finish(at, B("y"), p + "mix1"),
        ]

    def latent(i: int, at: int, prefill: bool) -> list[dict]:
        m, p = layers[i]["mixer"], f"l{i}."
        z = latent_sizes(m)
        H, dim, vdim, r, proj = m["heads"], m["dim"], m["vdim"], z["rank"], z["proj"]
        kv = f"kv.l{i}"
        states[kv] = {"bytes_per_token": r * es}
        room("proj", proj); room("qlat", z["lat"]); room("olat", z["lat"]); room("attn", z["v"]); room("y", d)
        w_in = weight(f"w.{p}mix.qgc", (proj, d), p + "mix.q", p + "mix.g", p + "mix.dkv",
                      *([{"tensor": p + "mix.q", "rows": [0, proj - z["rows"]]}] if proj > z["rows"] else []))
        app = op(f"latent_append_{r}x{proj}", lambda: K.latent_append_op(r, proj, cfg.eps, A))
        uk = same(p + "mix.uk", (z["q"], r))
        tiles = K.head_tiles(r, dim, proj, z["lat"], A)
        if tiles and prefill:      # the tensor-core form wants W_uk with a latent column per row: turned once, at load
            bufs[f"ukt.l{i}"] = {"dtype": "bf16", "shape": [H, r, dim], "kind": "carry"}
            once.append({"op": op(f"transpose_{H}x{dim}x{r}", lambda: K.transpose_heads_op(H, dim, r)), "label": p + "ukt", "args": [uk, B(f"ukt.l{i}")]})
        up = op(f"q_up_{H}x{dim}x{r}x{proj}", lambda: K.head_linear_op(H, r, dim, act=A, rows_max=T, lda=proj, ldc=z["lat"], transposed=not tiles))
        down = op(f"v_up_{H}x{vdim}x{r}", lambda: K.head_linear_op(H, vdim, r, act=A, rows_max=T, lda=z["lat"], ldc=z["v"]))
        gate = op(f"gate_{z['v']}x{proj}", lambda: K.gate_mul_op(z["v"], proj, A))
        sfx = "_p" if prefill else "_d"
        attn = op(f"latent_attn{sfx}_{H}x{r}x{m['scale']}", lambda: K.latent_attn_op(H, r, m["scale"], cfg.page_size, W, prefill, A, seqs_max=S))
        lens = [B("row_len"), err, B("row_seq")] if prefill else [B("seq_lens"), err]
        calls = [
            linear("lin", proj, d, B("xn"), w_in, B("proj"), label=p + "qgc"),
            {"op": app, "label": p + "append", "args": [B("proj", (z["q"] + z["v"]) * es), {"state": kv}, B("slot_mapping"),
                                                        same(p + "mix.dkv.norm", (r,))]},
            {"op": up, "label": p + "q_up", "args": [B("proj"), B(f"ukt.l{i}") if tiles else uk, B("qlat"), V("tokens"), err]},
            {"op": attn, "label": p + "attn", "args": [B("qlat"), {"state": kv}, B("olat"), B("block_table"), *lens]},
            {"op": down, "label": p + "v_up", "args": [B("olat"), same(p + "mix.uv", (z["v"], r)), B("attn"), V("tokens"), err]},
            {"op": gate, "label": p + "gate", "args": [B("attn"), B("proj", z["q"] * es), B("attn"), V("tokens")]},
            linear("lin", d, z["v"], B("attn"), same(p + "mix.o", (d, z["v"])), B("y"), label=p + "o"),
            finish(at, B("y"), p + "mix1"),
        ]
        if prefill and i == latents[0]:
            calls.insert(0, {"op": op("rows", C.mla_rows_op), "label": p + "rows", "args": [B("positions"), B("cu_seqlens"), B("row_seq"), B("row_len"), V("seqs"), V("tokens")]})
        return calls

    def dense(i: int, at: int) -> list[dict]:
        ff, p = layers[i]["mlp"]["ff"], f"l{i}."
        room("act", ff); room("y", d)
        return [
            linear("glu", 2 * ff, d, B("xn"), weight(f"w.{p}mlp.gu", (2 * ff, d), p + "mlp.gate", p + "mlp.up"), B("act"), label=p + "gate_up", epilogue="swiglu"),
            linear("lin", d, ff, B("act"), same(p + "mlp.down", (d, ff)), B("y"), label=p + "down"),
            finish(at, B("y"), p + "mix2"),
        ]

    def routed(i: int, at: int) -> list[dict]:
        f, p = layers[i]["mlp"], f"l{i}."
        E, k, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
        room("moe.logits", E, "f32"); room("moe.ids", k, "i32"); room("moe.w", k, "f32"); room("moe.perm", k, "i32")
        room("moe.x", k * d); room("moe.act", k * ff); room("moe.y", k * d)
        tiles = T * k // K.routed_tile_rows(A, d, ff) + E
        for name, shape in (("moe.offsets", [E + 1]), ("moe.tiles", [tiles, 4]), ("moe.tile_count", [1]), ("moe.rows", [1])):
            have = bufs.get(name, {"shape": [0]})["shape"]
            bufs[name] = {"dtype": "i32", "shape": [max(have[0], shape[0]), *shape[1:]], "kind": "workspace"}
        tag = f"{d}x{ff}x{E}x{k}"
        if f"moe_plan_{tag}" not in ops:
            for n, o in K.routed_ops(d, ff, E, k, T, A).items():
                ops[f"{n}_{tag}"] = o
        route = op(f"moe_route_{E}x{k}", lambda: K.route_logits_op(E, k))
        n = {"expr": {"mul": ["tokens", k]}}
        w1 = weight(f"w.{p}mlp.w1", (E, 2 * ff, d), *[f"{p}mlp.e{e}.{t}" for e in range(E) for t in ("gate", "up")])
        w2 = weight(f"w.{p}mlp.w2", (E, d, ff), *[f"{p}mlp.e{e}.down" for e in range(E)])
        return [
            linear("router", E, d, B("xn"), same(p + "mlp.router", (E, d)), B("moe.logits"), label=p + "router", epilogue="f32"),
            {"op": route, "label": p + "route", "args": [B("moe.logits"), same(p + "mlp.router.b", (E,)), B("moe.ids"), B("moe.w"), V("tokens")]},
            {"op": f"moe_plan_{tag}", "label": p + "plan", "args": [B("moe.ids"), B("moe.perm"), B("moe.offsets"), B("moe.tiles"), B("moe.tile_count"), B("moe.rows"), n, err]},
            {"op": f"moe_gather_{tag}", "label": p + "gather", "args": [B("xn"), B("moe.perm"), B("moe.x"), n]},
            {"op": f"moe_fc1_{tag}", "label": p + "fc1", "args": [B("moe.x"), w1, B("moe.act"), B("moe.tiles"), B("moe.tile_count"), n, err]},
            {"op": f"moe_fc2_{tag}", "label": p + "fc2", "args": [B("moe.act"), w2, B("moe.y"), B("moe.tiles"), B("moe.tile_count"), n, err]},
            finish(at, B("moe.y"), p + "mix2", k, [B("moe.perm"), B("moe.w")]),
        ]

    def forward(prefill: bool) -> list[dict]:
        embed = op("embed", lambda: K.hyper_embed_op(d, s, cfg.vocab, cfg.max_positions, cfg.eps, A))
        calls = [{"op": embed, "label": "embed", "args": [
            B("token_ids"), B("positions"), same("embed", (cfg.vocab, d)), same("pos", (cfg.max_positions, d)), same("embed.norm", (d,)),
            same(subs[0][0] + ".in", (s,)), same(subs[0][1], (d,)), B("x"), B("xn"), err]}]
        at = 0
        for i, b in enumerate(layers):
            calls += (mamba if kinds[i] == "mamba2" else latent)(i, at, prefill)
            at += 1
            if b["mlp"] is not None:
                calls += (dense if b["mlp"]["kind"] == "dense" else routed)(i, at)
                at += 1
        pick = "last" if prefill else "each"
        norm = op("final_norm_" + pick, lambda: K.row_norm_op(d, cfg.eps, T, A, pick))
        calls += [{"op": norm, "label": "final_norm", "args": [B("hidden"), same("final.norm", (d,)), B("last_n"), *([B("cu_seqlens")] if prefill else [])]},
                  linear("head", cfg.vocab, d, B("last_n"), same("head", (cfg.vocab, d)), B("logits"), rows="seqs", label="lm_head", epilogue="f32")]
        if cfg.sampling:
            pick_op = op("sample", lambda: C.sample_op(cfg.vocab, "f32"))
            calls.append({"op": pick_op, "label": "sample", "args": [B("logits"), B("next_token"), *[B(n) for n in
                          ("temperature", "top_k", "top_p", "min_p", "seed", "seq_lens")]]})
        else:
            calls.append({"op": op("pick", lambda: C.argmax_op(cfg.vocab, "f32")), "label": "argmax", "args": [B("logits"), B("next_token")]})
        return calls

    if cfg.sampling:
        bufs.setdefault("seq_lens", inp("i32", ["seqs"], fill="seq_len"))
        for name, dt in (("temperature", "f32"), ("top_k", "i32"), ("top_p", "f32"), ("min_p", "f32"), ("seed", "i64")):
            bufs[name] = inp(dt, ["seqs"], fill=name)
    prefill, decode = forward(True), forward(False)
    listed = op("final_norm_listed", lambda: K.row_norm_op(d, cfg.eps, T, A, "listed"))
    logits = [{"op": listed, "label": "want_norm", "args": [B("hidden"), B("w.final.norm"), B("want_n"), B("want_rows")]},
              linear("head_rows", cfg.vocab, d, B("want_n"), B("w.head"), B("want_logits"), rows="wanted", label="want_head", epilogue="f32")]
    doc = {
        "schema_version": 7, "model": cfg.name,
        "vars": {"tokens": {"max": T, "axis": "rows"}, "seqs": {"max": S, "axis": "groups"}, "wanted": {"max": WANTED}},
        "states": states, "buffers": bufs, "modules": {}, "ops": ops,
        "programs": {
            "prefill": {"batch": {"groups": S, "rows": "tokens"}, "calls": prefill},
            "decode": {"batch": {"groups": S, "rows": 1}, "graph": True, "calls": decode},
            "logits": {"calls": logits},
        },
    }
    if once:
        doc["programs"]["load"] = {"once": True, "calls": once}
    used = {l["module"] for o in ops.values() for l in o["impl"]["launches"]}
    doc["modules"] = {n: m for n, m in C.modules_for(sorted(used)).items() if n in used}
    return doc

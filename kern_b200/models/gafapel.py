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
from . import listed
from .listed import Listed, load_random


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
    load_random(rt, weight_names(cfg), _random, seed, std)


def save_folder(path, cfg: GafapelConfig, weights: dict[str, torch.Tensor]) -> None:
    listed.save_folder(path, to_config(cfg), weights)


# ---- the manifest -------------------------------------------------------------------------------------------
def build_manifest(cfg: GafapelConfig) -> dict:
    d, A, T, S, W = cfg.width, cfg.dtype, cfg.max_tokens, cfg.max_seqs, cfg.table_width
    m_ = Listed(cfg)
    layers, es, bufs, states, once, err = cfg.depth, m_.es, m_.bufs, m_.states, m_.once, m_.err
    B, V, op, room, weight, same, linear = m_.B, m_.V, m_.op, m_.room, m_.weight, m_.same, m_.linear
    kinds = [kind_of(b) for b in layers]
    latents = [i for i, k in enumerate(kinds) if k == "latent_attention"]
    mambas = [i for i, k in enumerate(kinds) if k == "mamba2"]
    m_.inputs(f"kv.l{latents[0]}" if latents else None, f"ssd.l{mambas[0]}" if mambas else None)
    room("x", cfg.streams * d, "f32")
    room("xn", d)
    m_.outputs()

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
            calls.insert(0, m_.rows_call(p + "rows"))
        return calls

    def dense(i: int, at: int) -> list[dict]:
        p = f"l{i}."
        return m_.dense(p, layers[i]["mlp"]["ff"], "swiglu") + [finish(at, B("y"), p + "mix2")]

    def routed(i: int, at: int) -> list[dict]:
        f, p = layers[i]["mlp"], f"l{i}."
        E, k = f["router"]["experts"], f["router"]["top"]
        route = op(f"moe_route_{E}x{k}", lambda: K.route_logits_op(E, k))
        pick = lambda logits, ids, w: {"op": route, "label": p + "route", "args": [logits, same(p + "mlp.router.b", (E,)), ids, w, V("tokens")]}
        return m_.routed(p, E, k, f["expert"]["ff"], pick) + [finish(at, B("moe.y"), p + "mix2", k, [B("moe.perm"), B("moe.w")])]

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
        return calls

    return m_.document(forward, "head")

"""Fusasun: a decoder whose layers are listed one by one. A layer's mixer is grouped-query attention in a sliding window that also sees
the mean key and value of every block of tokens before the window (rotary pairs of neighbours, frequencies scaled in bands), or
latent attention in a sliding window (queries through a latent, one rotated key part for all heads with YaRN frequencies, a gate per
head). Its feed-forward is experts that a table picks by the token id, or none. The mixer reads its input plus a short causal
convolution of it; every sublayer's result is gated element by element by its input, normed, and added.

Manifest generator, checkpoint names and synthetic weights. A layer owns a per-sequence line (the convolution's last inputs);
attention a paged state of its turned keys and its values and a second one, on the same pages, of the blocks' means; latent
attention one of its latents with the rotated part behind each. `dtype` "f32" is the exact form: every activation, cached row and
product in 32-bit over the same bf16 weights.

A program runs, per sublayer: mixer or feed-forward, and the gate's product, on the normed residual -> one kernel that gathers the
result (expert rows), gates, norms and adds it, makes the next sublayer's normed input and, one row per sequence, convolves it.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path

import torch

from . import blocks as K
from . import common as C
from . import listed
from .listed import Listed, latent_sizes, load_random


@dataclass
class FusasunConfig:
    name: str = "fusasun"
    width: int = 2304
    vocab: int = 163840
    eps: float = 1e-6
    taps: int = 4                                  # of the convolution before a mixer
    scale: float = 1.0                             # of the embedding
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
        return self.max_context or 8192

    @property
    def table_width(self) -> int:
        return -(-self.context // self.page_size)


_MIXER_KEYS = {"attention": {"dim": None, "heads": None, "kv_heads": None, "vdim": None, "scale": None, "mask": {"size", "pool"}, "rot": {"base", "dims"}},
               "latent_attention": {"dim": None, "heads": None, "kv_rank": None, "q_rank": None, "rot_dim": None, "vdim": None, "scale": None, "mask": {"size"},
                                    "rot": {"base", "dims"}}}
_SCALING_KEYS = {"attention": ("factor", "low", "high", "original"), "latent_attention": ("factor", "original", "fast", "slow")}


def _check_mixer(i: int, kind: str, m: dict) -> None:
    if kind not in _MIXER_KEYS:
        raise ValueError(f"layer {i}: unknown mixer `{kind}`; known: {', '.join(sorted(_MIXER_KEYS))}")
    missing = [k for k in _MIXER_KEYS[kind] if k not in m] + [f"{k}.{s}" for k, sub in _MIXER_KEYS[kind].items() if sub and k in m for s in sorted(sub - set(m[k]))]
    if not missing and m["rot"].get("scaling"):
        missing = [f"rot.scaling.{k}" for k in _SCALING_KEYS[kind] if k not in m["rot"]["scaling"]]
    if missing:
        raise ValueError(f"layer {i}: mixer `{kind}` lacks {missing}")
    if m["mask"]["size"] < 1 or m["mask"].get("pool", 1) < 1:
        raise ValueError(f"layer {i}: a window of {m['mask']['size']} positions, blocks of {m['mask'].get('pool')}")
    if kind == "latent_attention" and m["rot"]["dims"] != m["rot_dim"]:
        raise ValueError(f"layer {i}: {m['rot']['dims']} of {m['rot_dim']} rotated columns turn")


def _check_mlp(i: int, f: dict | None) -> None:
    if f is None:
        return
    if f.get("kind") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward `{f.get('kind')}`")
    missing = [k for k in ("expert", "router") if k not in f] or [k for k in ("experts", "top") if k not in f["router"]] + [k for k in ("ff",) if k not in f["expert"]]
    if missing:
        raise ValueError(f"layer {i}: experts lack {missing}")


def from_config(doc: dict, **over) -> FusasunConfig:
    """config.json -> the configuration; `over`: fields of the serving side (dtype, max_seqs, ..)."""
    for i, b in enumerate(doc["layers"]):
        _check_mixer(i, b["type"], b["mixer"])
        _check_mlp(i, b["mlp"])
    return FusasunConfig(name=over.pop("name", "fusasun"), width=doc["width"], vocab=doc["vocab"], eps=float(doc["norm"]["eps"]), taps=doc["canon"]["taps"],
                         scale=float(doc["embedding"]["scale"]), blocks=doc["layers"], **over)


def from_folder(path, **over) -> FusasunConfig:
    return from_config(json.loads((Path(path) / "config.json").read_text()), **over)


def to_config(cfg: FusasunConfig) -> dict:
    """The config.json of a configuration."""
    return {"architecture": "Fusasun", "canon": {"taps": cfg.taps}, "embedding": {"scale": cfg.scale}, "layers": cfg.depth, "norm": {"eps": cfg.eps}, "vocab": cfg.vocab,
            "width": cfg.width}


def _attention(heads, kv_heads, dim, vdim, window, pool, rot, base, bands, scale):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "pool": pool}, "scale": scale,
                         "rot": {"base": base, "dims": rot, "scaling": dict(zip(_SCALING_KEYS["attention"], bands))}}


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, base, yarn, scale):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
                                "scale": scale, "rot": {"base": base, "dims": rot_dim, "scaling": dict(zip(_SCALING_KEYS["latent_attention"], yarn))}}


def _block(mixer, mlp) -> dict:
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def _moe(experts: int, top: int, ff: int) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


TINY_FUSASUN = FusasunConfig(
    name="tiny-fusasun", width=128, vocab=256, page_size=16, max_tokens=256, max_seqs=8, max_context=512, taps=3, scale=1.5,
    blocks=[_block(_attention(4, 2, 64, 64, 40, 8, 32, 1e4, (4.0, 1.0, 4.0, 64), 0.125), _moe(9, 3, 40)),
            _block(_latent(5, 40, 24, 48, 96, 72, 30, 1e5, (2.0, 128, 16.0, 1.0), 0.12), _moe(6, 2, 56)),
            _block(_attention(6, 3, 48, 40, 25, 6, 16, 1e4, (8.0, 1.0, 2.0, 100), 0.15), None)])
# the width, depth, vocabulary and experts of the 48B-A3B shape class
FUSASUN_LARGE = FusasunConfig(
    name="fusasun-48b-a3b", width=2304, vocab=163840, scale=2.0,
    blocks=[_block(_latent(32, 128, 64, 128, 512, 1536, 1024, 1e6, (4.0, 4096, 32.0, 1.0), 192 ** -0.5) if i % 2 else
                   _attention(32, 4, 128, 128, 512, 16, 128, 5e5, (8.0, 1.0, 4.0, 8192), 128 ** -0.5), _moe(256, 8, 1024)) for i in range(27)])


# ---- sizes of a layer ---------------------------------------------------------------------------------------
def attention_sizes(m: dict) -> dict:
    return {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"], "o": m["heads"] * m["vdim"],
            "token": m["kv_heads"] * (m["dim"] + m["vdim"])}


def weight_names(cfg: FusasunConfig) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor name -> shape; the tables of experts are int32, everything else bf16."""
    d = cfg.width
    out = {"embed": (cfg.vocab, d)}
    for i, b in enumerate(cfg.depth):
        p, q, m, f = f"l{i}.", f"l{i}.mix.", b["mixer"], b["mlp"]
        out[p + "canon1"] = (d, cfg.taps)
        for n in "12" if f is not None else "1":
            out |= {f"{p}norm{n}": (d,), f"{p}norm{n}b": (d,), f"{p}rg{n}": (d, d), f"{p}rg{n}.b": (d,)}
        if b["type"] == "attention":
            z = attention_sizes(m)
            out |= {q + "q": (z["q"], d), q + "k": (z["k"], d), q + "v": (z["v"], d), q + "o": (d, z["o"])}
        else:
            z = latent_sizes(m)
            out |= {q + "dq": (m["q_rank"], d), q + "dq.norm": (m["q_rank"],), q + "uq": (z["q"] + z["rot"], m["q_rank"]), q + "dkv": (z["down"], d),
                    q + "dkv.norm": (z["rank"],), q + "uk": (z["q"], z["rank"]), q + "uv": (z["v"], z["rank"]), q + "g": (m["heads"], d), q + "o": (d, z["v"])}
        if f is not None:
            ff = f["expert"]["ff"]
            for e in range(f["router"]["experts"]):
                n = f"{p}mlp.e{e}."
                out |= {n + "gate": (ff, d), n + "up": (ff, d), n + "down": (d, ff)}
            out[p + "mlp.table"] = (cfg.vocab, f["router"]["top"])
    out |= {"final.norm": (d,), "head": (cfg.vocab, d)}
    return out


def random_table(vocab: int, top: int, experts: int, g, device) -> torch.Tensor:
    """Rows of different experts."""
    return torch.rand(vocab, experts, generator=g, device=device).argsort(-1)[:, :top].to(torch.int32).contiguous()


def _random_of(cfg: FusasunConfig):
    experts = {f"l{i}.mlp.table": b["mlp"]["router"]["experts"] for i, b in enumerate(cfg.depth) if b["mlp"] is not None}

    def make(name: str, shape, g, device, std: float) -> torch.Tensor:
        n = lambda: torch.randn(shape, generator=g, device=device)
        last = name.rsplit(".", 1)[-1]
        if name in experts:
            return random_table(*shape, experts[name], g, device)
        if "norm" in last:
            t = 1 + 0.1 * n()
        elif last == "canon1":
            t = 0.3 * n()
        elif last == "b":
            t = 0.5 * n()
        elif name == "embed":
            t = n()
        else:
            t = std * n()
        return t.to(torch.bfloat16)

    return make


def random_weights(cfg: FusasunConfig, seed: int = 0, device: str = "cpu", std: float = 0.02) -> dict[str, torch.Tensor]:
    g, make = torch.Generator(device=device).manual_seed(seed), _random_of(cfg)
    return {n: make(n, s, g, device, std) for n, s in weight_names(cfg).items()}


def load_random_weights(rt, cfg: FusasunConfig, seed: int = 0, std: float = 0.02) -> None:
    load_random(rt, weight_names(cfg), _random_of(cfg), seed, std)


def save_folder(path, cfg: FusasunConfig, weights: dict[str, torch.Tensor]) -> None:
    listed.save_folder(path, to_config(cfg), weights)


# ---- the manifest -------------------------------------------------------------------------------------------
def build_manifest(cfg: FusasunConfig) -> dict:
    d, A, S, W, page, eps = cfg.width, cfg.dtype, cfg.max_seqs, cfg.table_width, cfg.page_size, cfg.eps
    m_ = Listed(cfg)
    layers, es, states, err = cfg.depth, m_.es, m_.states, m_.err
    B, V, op, room, same, linear = m_.B, m_.V, m_.op, m_.room, m_.same, m_.linear
    tiled = {i: K.pooled_tiles(*(b["mixer"][k] for k in ("heads", "kv_heads", "dim", "vdim")), b["mixer"]["mask"]["pool"], page, A)
             for i, b in enumerate(layers) if b["type"] == "attention"}
    m_.inputs("kv.l0", "conv.l0", row_plan=any(not tiled.get(i) for i in range(len(layers))))
    room("x", d, "f32")
    room("xn", d)
    room("rg", d)
    m_.outputs()

    # every sublayer in order: its layer, and the suffix of its tensors
    subs = [(i, q) for i, b in enumerate(layers) for q in ((1, 2) if b["mlp"] is not None else (1,))]
    conv = lambda i, prefill: m_.input_conv(f"l{i}.canon1", cfg.taps, f"conv.l{i}", prefill)

    def gate(at: int) -> dict:
        i, q = subs[at]
        return linear("lin", d, d, B("xn"), same(f"l{i}.rg{q}", (d, d)), B("rg"), label=f"l{i}.rg{q}")

    def finish(at: int, y, label: str, prefill: bool, routed: int = 0, route=()) -> dict:
        """Sublayer `at`'s gated and normed result onto the residual; the next one's input, convolved where that is a mixer, or the
        residual itself after the last."""
        i, q = subs[at]
        post, g = same(f"l{i}.norm{q}b", (d,)), [B("rg"), same(f"l{i}.rg{q}.b", (d,))]
        if at + 1 == len(subs):
            name = op(f"resid_gate_last_{routed}", lambda: K.resid_gate_op(d, eps, A, routed, last=True))
            return {"op": name, "label": label, "args": [B("x"), y, post, B("hidden"), *g, *route]}
        ni, nq = subs[at + 1]
        args = [B("x"), y, post, same(f"l{ni}.norm{nq}", (d,)), B("xn"), *g, *route]
        if nq == 2:
            return {"op": op(f"resid_gate_{routed}", lambda: K.resid_gate_op(d, eps, A, routed)), "label": label, "args": args}
        c = conv(ni, prefill)
        if prefill:
            make = lambda: K.chain_ops(K.resid_gate_op(d, eps, A, routed), c["op"]())
        else:
            make = lambda: K.resid_gate_op(d, eps, A, routed, conv=c["fused"])
        return {"op": op(f"resid_gate_conv{'_p' if prefill else '_d'}_{routed}_{c['tag']}", make), "label": label, "args": args + c["args"]}

    def attention(i: int, prefill: bool) -> list[dict]:
        m, p, kv, means, sfx = layers[i]["mixer"], f"l{i}.mix.", f"kv.l{i}", f"pool.l{i}", "_p" if prefill else "_d"
        z, r, size, pool, scale = attention_sizes(m), m["rot"], m["mask"]["size"], m["mask"]["pool"], float(m["scale"])
        hq, hk, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        states[kv] = {"bytes_per_token": z["token"] * es}
        states[means] = {"bytes_per_token": K.pooled_sizes(hk, dim, vdim, pool, page, A)["token"]}
        w_in, qkv = m_.rows_weight(f"w.{p}qkv", d, [(p + "q", z["q"]), (p + "k", z["k"]), (p + "v", z["v"])])
        room("qkv", qkv); room("attn", z["o"]); room("y", d)
        s = r.get("scaling")
        tables = m_.rotary(r["dims"], float(r["base"]), scaling=C.banded_rope(*(float(s[k]) for k in _SCALING_KEYS["attention"])) if s else None)
        heads = f"{hq}x{hk}x{dim}x{vdim}"
        prep = op(f"prep_pool{sfx}_{heads}x{r['dims']}x{pool}x{qkv}", lambda: K.qk_prep_pool_op(hq, hk, dim, vdim, r["dims"], pool, page, W, qkv, cfg.context, prefill, A))
        attn = op(f"pooled_attn{sfx}_{heads}x{size}x{pool}x{qkv}_{scale!r}",
                  lambda: K.pooled_attn_op(hq, hk, dim, vdim, size, pool, scale, page, W, qkv, z["o"], prefill, A, seqs_max=S))
        lens, lists = B("seq_lens"), []
        if prefill and tiled[i]:
            lists = [B("cu_seqlens"), *m_.lists_of(hq, hk, dim)]
        elif prefill:
            lens, lists = B("row_len"), m_.row_plan()
        return [
            linear("lin", qkv, d, B("xc"), w_in, B("qkv"), label=p + "qkv"),
            {"op": prep, "label": p + "prep", "args": [B("qkv"), {"state": kv}, {"state": means}, B("positions"), B("slot_mapping"), B("block_table"), *tables, err,
                                                       *([B("cu_seqlens"), V("seqs"), V("tokens")] if prefill else [])]},
            {"op": attn, "label": p + "attn", "args": [B("qkv"), {"state": kv}, {"state": means}, B("attn"), B("block_table"), lens, err, *lists]},
            linear("lin", d, z["o"], B("attn"), same(p + "o", (d, z["o"])), B("y"), label=p + "o"),
        ]

    def latent(i: int, prefill: bool) -> list[dict]:
        m = layers[i]["mixer"]
        base, s = float(m["rot"]["base"]), m["rot"].get("scaling")
        scaling = C.ramped_rope(m["rot_dim"], base, *(float(s[k]) for k in _SCALING_KEYS["latent_attention"])) if s else None
        return m_.latent(f"l{i}.mix.", f"kv.l{i}", m, prefill, m_.rotary(m["rot_dim"], base, scaling=scaling), x="xc", halves=False, gate=True, window=m["mask"]["size"])

    mixers = {"attention": attention, "latent_attention": latent}

    def forward(prefill: bool) -> list[dict]:
        calls = []
        for at, (i, q) in enumerate(subs):
            p = f"l{i}."
            if q == 1:
                calls += [*mixers[layers[i]["type"]](i, prefill), gate(at), finish(at, B("y"), p + "mix.out", prefill)]
            else:
                r = layers[i]["mlp"]["router"]
                calls += [*m_.table_routed(p, r["experts"], r["top"], layers[i]["mlp"]["expert"]["ff"]), gate(at),
                          finish(at, B("moe.y"), p + "mlp.out", prefill, r["top"], [B("moe.perm"), B("moe.w")])]
        return [m_.embed("l0.norm1", prefill, cfg.scale, conv(0, prefill)), *calls]

    return m_.document(forward, "head")

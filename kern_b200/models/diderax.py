"""Diderax: a pre-norm decoder whose layers are listed one by one. A layer's mixer is grouped-query attention whose keys, as
projected, are its values (norms over whole projections, rotary halves with scaled frequencies, one added to the softmax
denominator, an output gate), latent attention (queries through a latent, one rotated key part for all heads, a sink per head),
or gated linear attention (a decay per key channel). Its feed-forward is a dense SwiGLU with biases, routed experts chosen inside
the best groups — some of which hand the input back — beside a gated shared one, or none. Every sublayer's result is scaled
element by element before it is added.

Manifest generator, checkpoint names and synthetic weights. Attention owns a paged state of its turned keys and its values, latent
attention one of its latents with the rotated part behind each, linear attention a per-sequence line of S in f32. `dtype` "f32"
is the exact form: every activation, cached row and product in 32-bit over the same bf16 weights.

A program runs, per sublayer: mixer or feed-forward on the normed residual -> one kernel that gathers the result (expert rows, the
input handed back, the shared expert, a bias), scales and adds it and makes the next sublayer's normed input. The rows of W_uq
are sorted when they are bound, the unrotated ones of all heads before the rotated ones.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path

import torch

from . import blocks as K
from . import common as C
from . import listed
from .listed import Listed, gla_sizes, latent_sizes, load_random


@dataclass
class DideraxConfig:
    name: str = "diderax"
    width: int = 2304
    vocab: int = 163840
    eps: float = 1e-6
    blocks: list = field(default_factory=list)     # the entries of config.json's `layers`
    ranks: list = field(default_factory=list)      # per layer: width of the decay's low-rank projection (a tensor's shape says it), or 0
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


_MIXER_KEYS = {"attention": {"dim", "heads", "kv_heads", "rot", "scale", "vdim"}, "gla": {"dim", "heads", "tau", "vdim"},
               "latent_attention": {"dim", "heads", "kv_rank", "q_rank", "rot", "rot_dim", "scale", "vdim"}}


def _check_mixer(i: int, kind: str, m: dict) -> None:
    if kind not in _MIXER_KEYS:
        raise ValueError(f"layer {i}: unknown mixer `{kind}`; known: {', '.join(sorted(_MIXER_KEYS))}")
    missing = _MIXER_KEYS[kind] - set(m)
    if not missing and "rot" in m:
        missing = {f"rot.{k}" for k in ("base", "dims") if k not in m["rot"]}
    if missing:
        raise ValueError(f"layer {i}: mixer `{kind}` lacks {sorted(missing)}")
    if kind == "attention" and m["vdim"] != m["dim"]:
        raise ValueError(f"layer {i}: keys of {m['dim']} columns are the values, of {m['vdim']}")
    if kind == "latent_attention" and m["rot"]["dims"] != m["rot_dim"]:
        raise ValueError(f"layer {i}: {m['rot']['dims']} of {m['rot_dim']} rotated columns turn")


def _check_mlp(i: int, f: dict | None) -> None:
    if f is None:
        return
    if f["kind"] not in ("dense", "moe"):
        raise ValueError(f"layer {i}: unknown feed-forward `{f['kind']}`")
    if f["kind"] == "moe":
        r = f["router"]
        missing = ({"experts", "top"} - set(r)) | ({"expert"} - set(f))
        if missing:
            raise ValueError(f"layer {i}: routed experts lack {sorted(missing)}")


def from_config(doc: dict, ranks: list[int], **over) -> DideraxConfig:
    """config.json and the decays' ranks -> the configuration; `over`: fields of the serving side (dtype, max_seqs, ..)."""
    for i, b in enumerate(doc["layers"]):
        _check_mixer(i, b["type"], b["mixer"])
        _check_mlp(i, b["mlp"])
    return DideraxConfig(name=over.pop("name", "diderax"), width=doc["width"], vocab=doc["vocab"], eps=float(doc["norm"]["eps"]), blocks=doc["layers"],
                         ranks=list(ranks), **over)


def from_folder(path, **over) -> DideraxConfig:
    doc = json.loads((Path(path) / "config.json").read_text())
    shapes = {}
    for f in sorted(Path(path).glob("*.safetensors")):
        shapes |= C.safetensors_shapes(f)
    return from_config(doc, [shapes[f"l{i}.mix.a1"][0] if b["type"] == "gla" else 0 for i, b in enumerate(doc["layers"])], **over)


def to_config(cfg: DideraxConfig) -> dict:
    """The config.json of a configuration."""
    return {"architecture": "Diderax", "layers": cfg.depth, "norm": {"eps": cfg.eps}, "vocab": cfg.vocab, "width": cfg.width}


def _attention(heads, kv_heads, dim, rot, base, factor, scale):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}}, "scale": scale}


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, base, scale):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                "rot": {"base": base, "dims": rot_dim}, "scale": scale}


def _gla(heads, dim, vdim, tau):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def _block(mixer, mlp) -> dict:
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def _dense(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def _moe(experts: int, identity: int, top: int, ff: int, groups: int, keep: int, scale: float, shared: int) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}}


TINY_DIDERAX = DideraxConfig(
    name="tiny-diderax", width=128, vocab=256, page_size=16, max_tokens=256, max_seqs=8, max_context=512,
    blocks=[_block(_gla(3, 24, 40, 8.0), _moe(9, 3, 3, 40, 3, 2, 1.5, 56)), _block(_attention(4, 2, 64, 32, 1e4, 4.0, 0.125), _dense(160)),
            _block(_latent(5, 40, 24, 48, 96, 72, 1e5, 0.12), _moe(9, 3, 3, 40, 3, 2, 1.5, 56)), _block(_attention(6, 3, 48, 16, 1e4, 2.0, 0.15), None)],
    ranks=[8, 0, 0, 0])
# the width, depth, vocabulary and experts of the 48B-A3B shape class; of four layers two are gated linear attention
_LARGE = [_gla(16, 128, 256, 16.0), _attention(32, 4, 128, 64, 1e6, 8.0, 128 ** -0.5), _gla(16, 128, 256, 16.0), _latent(32, 128, 64, 128, 512, 1536, 1e6, 192 ** -0.5)]
DIDERAX_LARGE = DideraxConfig(
    name="diderax-48b-a3b", width=2304, vocab=163840,
    blocks=[_block(_LARGE[i % 4], _dense(9216) if i == 1 else _moe(256, 8, 8, 1024, 8, 4, 2.5, 1024)) for i in range(27)], ranks=[0 if i % 2 else 64 for i in range(27)])


# ---- sizes of a layer ---------------------------------------------------------------------------------------
def attention_sizes(m: dict) -> dict:
    q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
    return {"q": q, "k": k, "token": 2 * k}


def moe_sizes(f: dict) -> dict:
    r = f["router"]
    identity, g = r.get("identity", 0), r.get("groups", {"count": 1, "keep": 1})
    return {"experts": r["experts"], "outputs": r["experts"] + identity, "top": r["top"], "groups": g["count"], "keep": g["keep"], "scale": float(r.get("scale", 1.0)),
            "shared": f["shared"]["ff"] if f.get("shared") else 0}


def weight_names(cfg: DideraxConfig) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor name -> shape; every tensor is bf16."""
    d = cfg.width
    out = {"embed": (cfg.vocab, d)}
    for i, b in enumerate(cfg.depth):
        p, q, m, f = f"l{i}.", f"l{i}.mix.", b["mixer"], b["mlp"]
        for n in "12" if f is not None else "1":
            out |= {f"{p}norm{n}": (d,), f"{p}ls{n}": (d,)}
        if b["type"] == "gla":
            z, rank = gla_sizes(m), cfg.ranks[i]
            out |= {q + "q": (z["q"], d), q + "k": (z["q"], d), q + "v": (z["v"], d), q + "g": (z["v"], d), q + "o": (d, z["v"]), q + "norm": (m["vdim"],),
                    q + "a1": (rank, d), q + "a2": (z["q"], rank), q + "a2.b": (z["q"],)}
        elif b["type"] == "attention":
            z = attention_sizes(m)
            out |= {q + "q": (z["q"], d), q + "k": (z["k"], d), q + "q.norm": (z["q"],), q + "k.norm": (z["k"],), q + "g": (z["q"], d), q + "o": (d, z["q"])}
        else:
            z = latent_sizes(m)
            out |= {q + "dq": (m["q_rank"], d), q + "dq.norm": (m["q_rank"],), q + "uq": (z["q"] + z["rot"], m["q_rank"]), q + "dkv": (z["down"], d),
                    q + "dkv.norm": (z["rank"],), q + "uk": (z["q"], z["rank"]), q + "uv": (z["v"], z["rank"]), q + "sink": (m["heads"],), q + "o": (d, z["v"])}
        if f is not None and f["kind"] == "dense":
            ff = f["ff"]
            out |= {p + "mlp.gate": (ff, d), p + "mlp.gate.b": (ff,), p + "mlp.up": (ff, d), p + "mlp.up.b": (ff,), p + "mlp.down": (d, ff), p + "mlp.down.b": (d,)}
        elif f is not None:
            z = moe_sizes(f)
            parts = [(f"{p}mlp.e{e}.", f["expert"]["ff"]) for e in range(z["experts"])] + ([(p + "mlp.shared.", z["shared"])] if z["shared"] else [])
            for n, ff in parts:
                out |= {n + "gate": (ff, d), n + "up": (ff, d), n + "down": (d, ff)}
            out |= {p + "mlp.router": (z["outputs"], d), p + "mlp.correction": (z["outputs"],)} | ({p + "mlp.shared.sg": (1, d)} if z["shared"] else {})
    out |= {"final.norm": (d,), "head": (cfg.vocab, d)}
    return out


def _random(name: str, shape, g, device, std: float) -> torch.Tensor:
    n = lambda: torch.randn(shape, generator=g, device=device)
    last = name.rsplit(".", 1)[-1]
    if "norm" in last:
        t = 1 + 0.1 * n()
    elif last in ("ls1", "ls2"):
        t = 0.5 + 0.1 * n()
    elif name.endswith("a2.b"):
        t = 2 + n()
    elif last == "b":
        t = 0.1 * n()
    elif last == "sink":
        t = n()
    elif last == "correction":
        t = 0.05 * n() / shape[0]               # of the size of a score's deviations
    elif last == "router":
        t = 10 * std * n()                      # a router with opinions
    elif name == "embed":
        t = n()
    else:
        t = std * n()
    return t.to(torch.bfloat16)


def random_weights(cfg: DideraxConfig, seed: int = 0, device: str = "cpu", std: float = 0.02) -> dict[str, torch.Tensor]:
    g = torch.Generator(device=device).manual_seed(seed)
    return {n: _random(n, s, g, device, std) for n, s in weight_names(cfg).items()}


def load_random_weights(rt, cfg: DideraxConfig, seed: int = 0, std: float = 0.02) -> None:
    load_random(rt, weight_names(cfg), _random, seed, std)


def save_folder(path, cfg: DideraxConfig, weights: dict[str, torch.Tensor]) -> None:
    listed.save_folder(path, to_config(cfg), weights)


# ---- the manifest -------------------------------------------------------------------------------------------
def build_manifest(cfg: DideraxConfig) -> dict:
    d, A, S, W, page, eps = cfg.width, cfg.dtype, cfg.max_seqs, cfg.table_width, cfg.page_size, cfg.eps
    m_ = Listed(cfg)
    layers, es, bufs, states, err = cfg.depth, m_.es, m_.bufs, m_.states, m_.err
    B, V, op, room, weight, same, linear = m_.B, m_.V, m_.op, m_.room, m_.weight, m_.same, m_.linear
    kinds = [b["type"] for b in layers]
    paged = [i for i, k in enumerate(kinds) if k != "gla"]
    lined = [i for i, k in enumerate(kinds) if k == "gla"]
    tiled = {i: K.window_tiles(*(layers[i]["mixer"][k] for k in ("heads", "kv_heads", "dim", "vdim")), page, A) for i in paged if kinds[i] == "attention"}
    m_.inputs(f"kv.l{paged[0]}" if paged else None, f"lin.l{lined[0]}" if lined else None, positions=bool(paged), row_plan=any(not tiled.get(i) for i in paged))
    room("x", d, "f32")
    room("xn", d)
    m_.outputs()

    # every sublayer in order: its norm, its scale
    subs = [(f"l{i}.norm{q}", f"l{i}.ls{q}") for i, b in enumerate(layers) for q in ((1, 2) if b["mlp"] is not None else (1,))]

    def finish(at: int, y, label: str, bias=None, routed: int = 0, route=(), shared_gate: int | None = None, shared=()) -> dict:
        """Sublayer `at`'s scaled result onto the residual; the next one's input, or the residual itself after the last."""
        last = at + 1 == len(subs)
        tag = f"{'last' if last else 'scale'}_{routed}" + ("_bias" if bias else "") + (f"_shared{shared_gate}" if shared else "")
        name = op("resid_" + tag, lambda: K.resid_scale_op(d, eps, A, routed=routed, bias=bool(bias), shared_gate=shared_gate, last=last))
        tail = [B("hidden")] if last else [same(subs[at + 1][0], (d,)), B("xn")]
        extra = [*([bias] if bias else []), *route, *shared, *([B("xn")] if last and routed else [])]
        return {"op": name, "label": label, "args": [B("x"), y, same(subs[at][1], (d,)), *tail, *extra]}

    def gla(i: int, at: int, prefill: bool) -> list[dict]:
        p = f"l{i}.mix."
        return m_.gla(p, f"lin.l{i}", layers[i]["mixer"], cfg.ranks[i], prefill) + [finish(at, B("y"), p + "out")]

    def attention(i: int, at: int, prefill: bool) -> list[dict]:
        m, p, kv, sfx = layers[i]["mixer"], f"l{i}.mix.", f"kv.l{i}", "_p" if prefill else "_d"
        z, r = attention_sizes(m), m["rot"]
        hq, hk, dim, q, k = m["heads"], m["kv_heads"], m["dim"], z["q"], z["k"]
        states[kv] = {"bytes_per_token": z["token"] * es}
        w_in, qkg = m_.rows_weight(f"w.{p}qkg", d, [(p + "q", q), (p + "k", k), (p + "g", q)])
        room("qkg", qkg); room("attn", q); room("y", d)
        cos_sin = m_.rotary(r["dims"], float(r["base"]), float((r.get("scaling") or {}).get("factor", 1.0)))
        prep = op(f"prep_whole_{hq}x{hk}x{dim}x{r['dims']}x{qkg}", lambda: K.qk_prep_whole_op(hq, hk, dim, dim, q, r["dims"], page, qkg, cfg.context, eps, A, halves=True))
        attn = op(f"sink_attn{sfx}_{hq}x{hk}x{dim}x{qkg}_{m['scale']!r}", lambda: K.sink_attn_op(hq, hk, dim, dim, float(m["scale"]), page, W, qkg, q, qkg, prefill, A, seqs_max=S))
        lens, lists = B("seq_lens"), []
        if prefill and tiled[i]:
            lists = [B("cu_seqlens"), *m_.lists_of(hq, hk, dim)]
        elif prefill:
            lens, lists = B("row_len"), m_.row_plan()
        return [
            linear("lin", qkg, d, B("xn"), w_in, B("qkg"), label=p + "qkg"),
            {"op": prep, "label": p + "prep", "args": [B("qkg"), {"state": kv}, B("positions"), B("slot_mapping"), *cos_sin, same(p + "q.norm", (q,)),
                                                       same(p + "k.norm", (k,)), err]},
            {"op": attn, "label": p + "attn", "args": [B("qkg"), {"state": kv}, B("attn"), B("block_table"), lens, B("qkg", (q + k) * es), err, *lists]},
            linear("lin", d, q, B("attn"), same(p + "o", (d, q)), B("y"), label=p + "o"),
            finish(at, B("y"), p + "out"),
        ]

    def latent(i: int, at: int, prefill: bool) -> list[dict]:
        m, p = layers[i]["mixer"], f"l{i}.mix."
        return m_.latent(p, f"kv.l{i}", m, prefill, m_.rotary(m["rot_dim"], float(m["rot"]["base"])), sink=True) + [finish(at, B("y"), p + "out")]

    def dense(i: int, at: int) -> list[dict]:
        p = f"l{i}."
        return m_.dense(p, layers[i]["mlp"]["ff"], "swiglu", bias=True) + [finish(at, B("y"), p + "mlp.out", bias=same(p + "mlp.down.b", (d,)))]

    def routed(i: int, at: int) -> list[dict]:
        f, p = layers[i]["mlp"], f"l{i}."
        z = moe_sizes(f)
        E, n, k = z["experts"], z["outputs"], z["top"]
        # the shared expert's gate is one more row of the router
        router = m_.rows_weight(f"w.{p}mlp.router", d, [(p + "mlp.router", n)] + ([(p + "mlp.shared.sg", 1)] if z["shared"] else []))
        ld = router[1]
        route = op(f"moe_route_{n}x{k}_{z['keep']}of{z['groups']}_{ld}_{z['scale']!r}", lambda: K.route_groups_op(
            n, k, z["groups"], z["keep"], True, softmax=True, correction=True, group_top=1, scale=z["scale"], ld=ld))
        pick = lambda logits, ids, w: {"op": route, "label": p + "route", "args": [logits, same(p + "mlp.correction", (n,)), ids, w, V("tokens")]}
        shared = {"shared_gate": ld, "shared": [B("shared.y"), B("moe.logits", n * 4)]} if z["shared"] else {}
        return m_.routed(p, E, k, f["expert"]["ff"], pick, router=router) + (m_.shared(p, z["shared"]) if z["shared"] else []) \
            + [finish(at, B("moe.y"), p + "mlp.out", routed=k, route=[B("moe.perm"), B("moe.w")], **shared)]

    mixers = {"gla": gla, "attention": attention, "latent_attention": latent}

    def forward(prefill: bool) -> list[dict]:
        calls, at = [], 0
        for i, b in enumerate(layers):
            calls += mixers[kinds[i]](i, at, prefill)
            at += 1
            if b["mlp"] is not None:
                calls += (dense if b["mlp"]["kind"] == "dense" else routed)(i, at)
                at += 1
        return [m_.embed(subs[0][0], prefill), *calls]

    return m_.document(forward, "head")

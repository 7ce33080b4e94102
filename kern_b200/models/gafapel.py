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

"""Small Fusasun configurations and the machinery that holds an engine against the plain oracle."""
import torch

from kern_b200.engine import Engine
from kern_b200.models import fusasun as G
from tests.barotar_cases import LIMIT  # noqa: F401
from tests.gafapel_cases import block, error, errors, play, portions, prompts_of, schedules  # noqa: F401
from tests.oracles import fusasun as O


def attention(heads, kv_heads, dim, vdim, window, pool, rot, base, bands, scale):
    return "attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window, pool=pool), scale=scale,
                             rot=dict(base=base, dims=rot, scaling=dict(zip(("factor", "low", "high", "original"), bands))))


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, base, yarn, scale):
    return "latent_attention", dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, mask=dict(size=window), scale=scale,
                                    rot=dict(base=base, dims=rot_dim, scaling=dict(zip(("factor", "original", "fast", "slow"), yarn))))


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


CASES = {
    # aligned sizes on the tensor-core tiles, two attention sizes with tiles of their own
    "mixed": dict(width=72, vocab=200, eps=1e-5, taps=4, scale=1.5, blocks=[
        block(attention(4, 2, 64, 64, 20, 8, 32, 1e4, (4.0, 1.0, 4.0, 64), 0.2), moe(9, 3, 24)), block(latent(5, 24, 16, 40, 72, 56, 13, 1e4, (2.0, 40, 8.0, 1.0), 0.3), moe(6, 2, 32)),
        block(attention(4, 1, 128, 128, 9, 16, 128, 5e5, (8.0, 1.0, 4.0, 30), 0.1)), block(latent(3, 16, 32, 24, 128, 40, 40, 1e5, (4.0, 100, 16.0, 2.0), 0.25), moe(4, 1, 48))]),
    # nothing is a multiple of eight, blocks that do not fit pages, more experts per token than not
    "odd": dict(width=50, vocab=101, eps=1e-6, taps=3, scale=0.7, blocks=[
        block(latent(3, 14, 6, 10, 36, 22, 17, 100.0, (3.0, 30, 4.0, 1.0), 0.5), moe(5, 4, 30)), block(attention(6, 2, 18, 10, 11, 6, 6, 300.0, (2.0, 0.5, 3.0, 25), 0.4)),
        block(attention(3, 1, 40, 72, 7, 24, 40, 1e4, (8.0, 1.0, 4.0, 100), 0.25), moe(3, 1, 11))]),
    # windows and blocks of one token, one never filled; no past in the convolution; sixteen heads and more, a head dim of 256
    "edges": dict(width=64, vocab=120, eps=1e-6, taps=1, scale=3.0, blocks=[
        block(latent(17, 8, 64, 16, 128, 24, 1, 1e6, (4.0, 512, 32.0, 1.0), 0.25), moe(3, 2, 16)), block(attention(3, 3, 256, 256, 1, 4, 64, 1e6, (2.0, 1.0, 4.0, 64), 0.08)),
        block(attention(2, 2, 64, 64, 600, 4, 2, 1e3, (5.0, 1.0, 2.0, 16), 0.15)), block(attention(4, 2, 64, 64, 12, 1, 64, 1e4, (1.0, 1.0, 4.0, 64), 0.2), moe(2, 2, 24))]),
    # a long convolution, blocks of several pages, a head group of sixteen, all layers without feed-forward but one
    "long": dict(width=96, vocab=160, eps=1e-4, taps=7, scale=1.0, blocks=[
        block(attention(16, 1, 64, 64, 5, 32, 64, 1e4, (8.0, 1.0, 4.0, 32), 0.15)), block(latent(2, 16, 8, 8, 56, 8, 64, 1e4, (8.0, 64, 4.0, 1.0), 0.4), moe(4, 2, 16)),
        block(attention(12, 4, 40, 40, 16, 16, 40, 1e4, (1.5, 1.0, 4.0, 50), 0.25))]),
}


def config(name, dtype="bf16", **over):
    return G.FusasunConfig(**{**dict(name=name, max_context=1200, page_size=16, max_tokens=160, max_seqs=12, dtype=dtype), **CASES[name], **over})


def weights(cfg, seed=0):
    """Random weights at which every layer speaks up: unit-scale projections, and queries far enough apart to pick keys."""
    w = G.random_weights(cfg, seed=seed, std=1.0)
    for n, t in w.items():
        if t.dim() == 2 and not n.endswith((".table", ".canon1")) and n != "embed":
            gain = 2.0 if n.endswith((".rg1", ".rg2", ".mix.g")) else (1.8 if n.endswith((".uq", ".uk", ".mix.q", ".mix.k")) else 1.0)
            w[n] = (t.float() * gain / t.shape[1] ** 0.5).to(torch.bfloat16)
    return w


def within(rows, dtype: str) -> bool:
    """No router decides anything here, so bf16 is held to its limit in every row, with room for the odd large one."""
    if dtype == "f32":
        return float(rows.max()) < LIMIT["f32"]
    return float(rows.quantile(0.9)) < LIMIT["bf16"] and float(rows.max()) < 3 * LIMIT["bf16"]


def engine(cfg, w, gpu: bool, tokens=None, slots=4):
    doc = G.build_manifest(cfg)
    tokens = tokens or 40 * cfg.page_size
    if gpu:
        from kern_b200.runtime import Runtime

        rt = Runtime(doc, tokens=tokens, slots=slots, guard_bands=True)
        rt.load_tensors(lambda n: w[n].cuda())
    else:
        from kern_b200.cpu import CpuRuntime

        rt = CpuRuntime(doc, weights=w, tokens=tokens, slots=slots)
    rt.once()
    return Engine(rt)


class Truth:
    """The oracle's logits of whole sequences."""

    def __init__(self, cfg, w):
        self.model = O.Model(G.to_config(cfg), w)
        self.kept = {}

    def __call__(self, ids):
        key = tuple(ids)
        if key not in self.kept:
            self.kept[key] = self.model.forward(list(ids), self.model.new_cache())
        return self.kept[key]

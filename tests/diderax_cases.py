"""Small Diderax configurations and the machinery that holds an engine against the plain oracle."""
import dataclasses

import torch

from kern_b200.engine import Engine
from kern_b200.models import diderax as G
from tests.barotar_cases import LIMIT, gla, within  # noqa: F401
from tests.gafapel_cases import block, dense, error, errors, play, portions, prompts_of, run_op, schedules  # noqa: F401
from tests.oracles import diderax as O


def attention(heads, kv_heads, dim, rot, base, factor, scale):
    return "attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, rot=dict(base=base, dims=rot, scaling=dict(factor=factor)), scale=scale)


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, base, scale):
    return "latent_attention", dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, rot=dict(base=base, dims=rot_dim), scale=scale)


def moe(experts, identity, top, ff, groups, keep, scale, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}}


CASES = {
    # aligned sizes on the tensor-core tiles, every branch, two attention sizes with tiles of their own
    "mixed": dict(width=72, vocab=200, eps=1e-5, ranks=[0, 16, 0, 0, 8], blocks=[
        block(attention(4, 2, 64, 32, 1e4, 3.0, 0.2), moe(9, 3, 3, 24, 4, 2, 1.7, 40)), block(gla(3, 40, 24, 4.0), dense(88)),
        block(latent(5, 24, 16, 40, 72, 56, 1e4, 0.3), moe(6, 2, 2, 32, 2, 1, 0.6, 16)),
        block(attention(4, 1, 128, 128, 5e5, 8.0, 0.1)), block(gla(2, 16, 72, 16.0), dense(48))]),
    # nothing is a multiple of eight, one group per output, more experts that hand back the input than others
    "odd": dict(width=50, vocab=101, eps=1e-6, ranks=[0, 3, 0], blocks=[
        block(latent(3, 14, 6, 10, 36, 22, 100.0, 0.5), moe(2, 3, 2, 30, 5, 3, 2.5, 11)), block(gla(3, 5, 33, 1.0)),
        block(attention(6, 2, 18, 6, 300.0, 1.0, 0.4), dense(30))]),
    "states_only": dict(width=64, vocab=96, eps=1e-6, ranks=[16, 4], blocks=[block(gla(2, 130, 20, 8.0)), block(gla(4, 17, 136, 2.0), moe(4, 4, 1, 24, 1, 1, 1.0, 8))]),
    # a latent that fills its blocks so that the rotated part has one to itself, sixteen heads and more, a head dim of 256,
    # a last feed-forward that hands back its input
    "edges": dict(width=64, vocab=120, eps=1e-6, ranks=[0, 0, 0], blocks=[
        block(latent(17, 8, 64, 16, 128, 24, 1e6, 0.25), dense(40)), block(attention(3, 3, 256, 64, 1e6, 2.0, 0.08)),
        block(latent(2, 16, 8, 8, 56, 8, 1e4, 0.4), moe(3, 1, 2, 16, 2, 2, 3.0, 24))]),
    "heads": dict(width=96, vocab=160, eps=1e-4, ranks=[0, 0, 5], blocks=[
        block(attention(16, 1, 64, 2, 1e3, 5.0, 0.15)), block(attention(12, 4, 40, 40, 1e4, 1.5, 0.25), moe(12, 0, 4, 16, 3, 2, 1.0, 8)), block(gla(1, 64, 64, 32.0))]),
}


def config(name, dtype="bf16", **over):
    return G.DideraxConfig(**{**dict(name=name, max_context=1200, page_size=16, max_tokens=160, max_seqs=12, dtype=dtype), **CASES[name], **over})


def decided(cfg):
    """The same model with every expert of a layer chosen: in bf16 a close call of a random router goes either way, and a state
    carries it on."""
    def every(m):
        r = m["router"]
        return {**m, "router": {**r, "top": r["experts"] + r["identity"], "groups": {**r["groups"], "keep": r["groups"]["count"]}}}

    return dataclasses.replace(cfg, blocks=[b if not b["mlp"] or b["mlp"]["kind"] == "dense" else {**b, "mlp": every(b["mlp"])} for b in cfg.blocks])


def weights(cfg, seed=0):
    """Random weights at which every layer speaks up: unit-scale projections, and queries far enough apart to pick keys."""
    w = G.random_weights(cfg, seed=seed, std=1.0)
    for n, t in w.items():
        if n.endswith("correction"):
            w[n] = (t.float() * 8).to(torch.bfloat16)                # some choices go below zero
        elif n.endswith((".gate.b", ".up.b", ".down.b")):
            w[n] = (t.float() * 5).to(torch.bfloat16)
        elif t.dim() == 2 and n != "embed":
            gain = 3.0 if n.endswith("router") else (1.5 if n.endswith((".uq", ".uk")) else 1.0)
            w[n] = (t.float() * gain / t.shape[1] ** 0.5 / (10.0 if n.endswith("router") else 1.0)).to(torch.bfloat16)
        elif n.endswith(".q.norm"):
            w[n] = (t.float() * 2.0).to(torch.bfloat16)
    return w


def engine(cfg, w, gpu: bool, tokens=None, slots=4):
    doc = G.build_manifest(cfg)
    tokens = tokens or 40 * cfg.page_size
    slots = slots if any(s.get("bytes_per_seq") for s in doc["states"].values()) else 0
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

"""Small Barotar configurations and the machinery that holds an engine against the plain oracle."""
import dataclasses

import torch

from kern_b200.engine import Engine
from kern_b200.models import barotar as G
from tests.gafapel_cases import block, dense, error, errors, play, portions, prompts_of, run_op, schedules  # noqa: F401
from tests.oracles import barotar as O


def gla(heads, dim, vdim, tau):
    return "gla", dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def parallel(left, right, left_scale, right_scale):
    """left: (heads, kv_heads, dim, vdim, window, rotated columns, base, scale, cap); right: (heads, dim)."""
    h, g, d, e, size, rot, base, scale, cap = left
    return "parallel", dict(left=dict(heads=h, kv_heads=g, dim=d, vdim=e, mask=dict(size=size), rot=dict(base=base, dims=rot), scale=scale, softcap=cap),
                            right=dict(heads=right[0], dim=right[1]), left_scale=left_scale, right_scale=right_scale)


def moe(experts, top, ff, groups, keep, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


CASES = {
    # aligned sizes on the tensor-core tiles, every branch, two attention sizes with tiles of their own
    "mixed": dict(width=72, vocab=200, eps=1e-5, ranks=[8, 16, 24, 8], blocks=[
        block(parallel((4, 2, 64, 64, 21, 32, 1e4, 0.15, 9.0), (3, 24), 0.7, 1.2), moe(12, 3, 24, 3, 2, 1.5)),
        block(gla(3, 40, 24, 4.0), dense(88)),
        block(parallel((4, 1, 128, 128, 50, 128, 5e5, 0.1, 28.0), (2, 64), 1.3, 0.4)),
        block(gla(2, 16, 72, 16.0), moe(8, 2, 32, 2, 1, 0.8))]),
    # nothing is a multiple of eight, keys and values of different sizes, one group per expert
    "odd": dict(width=50, vocab=101, eps=1e-6, ranks=[5, 3, 7], blocks=[
        block(parallel((6, 2, 18, 11, 9, 6, 100.0, 0.4, 5.0), (5, 7), 0.5, 1.0), moe(5, 2, 30, 5, 3, 2.5)),
        block(gla(3, 5, 33, 1.0)),
        block(parallel((3, 3, 14, 22, 33, 14, 1e3, 0.3, 50.0), (2, 13), 1.0, 0.8), dense(30))]),
    "states_only": dict(width=64, vocab=96, eps=1e-6, ranks=[16, 4], blocks=[block(gla(2, 130, 20, 8.0)), block(gla(4, 17, 136, 2.0), dense(48))]),
    # a window of one token, one that no sequence fills, a head dim of 256
    "edges": dict(width=64, vocab=120, eps=1e-6, ranks=[8, 8, 8], blocks=[
        block(parallel((2, 1, 64, 64, 1, 2, 1e4, 0.2, 20.0), (1, 64), 1.0, 1.0), dense(40)),
        block(parallel((3, 3, 256, 256, 700, 64, 1e6, 0.06, 12.0), (4, 16), 2.0, 0.3), moe(6, 6, 16, 1, 1, 3.0)),
        block(parallel((16, 1, 128, 128, 64, 64, 1e4, 0.1, 15.0), (2, 32), 1.1, 0.9))]),
}


def config(name, dtype="bf16", **over):
    return G.BarotarConfig(**{**dict(name=name, max_context=1200, page_size=16, max_tokens=160, max_seqs=12, dtype=dtype), **CASES[name], **over})


def decided(cfg):
    """The same model with every expert of a layer chosen: in bf16 a close call of a random router goes either way, and a state
    carries it on."""
    def every(m):
        return moe(m["router"]["experts"], m["router"]["experts"], m["expert"]["ff"], m["router"]["groups"]["count"], m["router"]["groups"]["count"], m["expert"]["limit"])

    return dataclasses.replace(cfg, blocks=[b if not b["mlp"] or b["mlp"]["kind"] == "dense" else {**b, "mlp": every(b["mlp"])} for b in cfg.blocks])


def weights(cfg, seed=0):
    """Random weights at which every layer speaks up: unit-scale projections, and queries far enough apart to pick keys."""
    w = G.random_weights(cfg, seed=seed, std=1.0)
    for n, t in w.items():
        if t.dim() == 2 and n != "embed" and not n.endswith(".u"):
            gain = 3.0 if n.endswith("router") else 1.0
            w[n] = (t.float() * gain / t.shape[1] ** 0.5 / (10.0 if n.endswith("router") else 1.0)).to(torch.bfloat16)
        elif n.endswith(".q.norm"):
            w[n] = (t.float() * 2.5).to(torch.bfloat16)
    return w


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


LIMIT = {"f32": 2e-4, "bf16": 8e-2}


def within(rows, dtype: str) -> bool:
    """f32: every row. bf16: all but a tenth (a head whose first tokens nearly cancel is normed up, rounding and all), and those
    not wild."""
    if dtype == "f32":
        return float(rows.max()) < LIMIT["f32"]
    return float(rows.quantile(0.9)) < LIMIT["bf16"] and float(rows.max()) < 0.7


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

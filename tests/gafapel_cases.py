"""Small Gafapel configurations and the machinery that holds an engine, or one op, against the plain oracle."""
import random

import torch

from kern_b200.engine import Engine
from kern_b200.models import common as C
from kern_b200.models import gafapel as G
from kern_b200.replay import Replay
from tests.oracles import gafapel as O


def mamba(heads, vdim, state, groups, conv, parts, kind="mamba2"):
    return kind, dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=parts)


def latent(heads, dim, vdim, rank, scale):
    return "latent_attention", dict(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, scale=scale)


def block(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


CASES = {
    # aligned sizes (tensor-core tiles), a head count that leaves the projection's rows ragged, every branch
    "mixed": dict(width=72, vocab=200, streams=3, eps=1e-5, blocks=[
        block(mamba(6, 20, 24, 3, 2, 4), dense(88)), block(latent(5, 24, 40, 72, 0.3), moe(10, 3, 24)),
        block(mamba(4, 16, 40, 1, 4, 1, "mamba2_2"), moe(6, 1, 32)), block(latent(2, 16, 16, 136, 0.11))]),
    # nothing is a multiple of eight
    "odd": dict(width=50, vocab=101, streams=1, eps=1e-6, blocks=[
        block(latent(3, 14, 10, 36, 0.5), moe(4, 4, 30)), block(mamba(3, 5, 7, 1, 5, 3), dense(30)),
        block(mamba(9, 7, 33, 3, 1, 7, "mamba2_2"), moe(5, 2, 11))]),
    "states_only": dict(width=64, vocab=96, streams=5, eps=1e-6, blocks=[block(mamba(4, 17, 130, 2, 3, 2)), block(mamba(2, 64, 16, 2, 4, 8), dense(48))]),
    # ragged width, aligned latents: per-head products on the tiles, everything else generic
    "ragged_width": dict(width=60, vocab=99, streams=2, eps=1e-6, blocks=[block(latent(3, 16, 24, 40, 0.3), dense(36)), block(mamba(2, 8, 20, 1, 3, 1))]),
    "cache_only": dict(width=96, vocab=160, streams=2, eps=1e-6, blocks=[block(latent(20, 8, 16, 200, 0.4), dense(64)), block(latent(17, 32, 8, 64, 0.2))]),
}


def config(name, dtype="bf16", **over):
    return G.GafapelConfig(**{**dict(name=name, max_positions=1200, page_size=16, max_tokens=160, max_seqs=8, dtype=dtype), **CASES[name], **over})


def weights(cfg, seed=0):
    """Random weights at which every layer speaks up: unit-scale projections and queries far enough apart to pick keys."""
    w = G.random_weights(cfg, seed=seed, std=1.0)
    for n, t in w.items():
        if t.dim() == 2 and n not in ("embed", "pos") and ".hc" not in n and not n.endswith(".conv"):
            gain = 2.0 if n.endswith((".q", ".uk")) else (3.0 if n.endswith("router") else 1.0)
            w[n] = (t.float() * gain / t.shape[1] ** 0.5 / (10.0 if n.endswith("router") else 1.0)).to(torch.bfloat16)
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


def errors(got, want):
    """Per row: root mean square of the difference without its mean, over the spread of the expected logits."""
    d = torch.as_tensor(got).double() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std(-1).clamp_min(1e-6)


def error(got, want):
    return float(errors(got, want).max())


def within(rows, dtype: str) -> bool:
    """f32: every row. bf16: all but a tenth (a random router has close calls that rounding decides), and those not wild."""
    if dtype == "f32":
        return float(rows.max()) < LIMIT["f32"]
    return float(rows.quantile(0.9)) < LIMIT["bf16"] and float(rows.max()) < 0.7


LIMIT = {"f32": 2e-4, "bf16": 6e-2}


def play(eng, truth, prompts, schedule):
    """`schedule`: steps of [(request, count), ..]; a request that reaches its prompt's end is given back, and named again
    it starts over. Every position's logits are asked for. -> the errors of all positions."""
    run, at, seen = Replay(eng), {}, []
    live = {}
    for step in schedule:
        entries, end, want = [], [], []
        for r, n in step:
            lo = at.get(r, 0)
            if lo == 0:
                live[r] = f"{r}.{random.random()}"
            toks = prompts[r][lo:lo + n]
            entries.append({"id": live[r], "tokens": toks, "want": list(range(len(toks)))})
            want.append(truth(prompts[r])[lo:lo + len(toks)])
            at[r] = lo + len(toks)
            if at[r] == len(prompts[r]):
                end.append(live[r])
                at[r] = 0
        seen.append(errors(run.step(entries, end), torch.cat(want)))
    assert not run.live, "the schedule ends every request"
    assert eng.pool.free_pages == eng.pool.total_pages and eng.pool.free_slots == eng.pool.total_slots
    return torch.cat(seen)


def portions(total, sizes):
    out, i = [], 0
    while sum(out) < total:
        out.append(min(sizes[i % len(sizes)], total - sum(out)))
        i += 1
    return out


def prompts_of(cfg, lengths, seed=1):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, cfg.vocab, (n,), generator=g).tolist() for i, n in enumerate(lengths)}


def schedules(prompts, page):
    """name -> schedule over four requests."""
    names, length = list(prompts), {r: len(p) for r, p in prompts.items()}
    out = {"whole": [[(r, length[r])] for r in names],
           "one_by_one": [[(names[0], 1)]] * length[names[0]],
           "whole_then_decode": [s for r in names for s in [[(r, max(1, length[r] - 9))]] + [[(r, 1)]] * min(9, length[r] - 1)],
           "portions": [[(r, n)] for r in names for n in portions(length[r], [2, page, 3, page - 1, 2, 1, page + 1])]}
    # all at once, unequal portions beside single tokens; then the same requests again on the pages and slots given back
    mixed = []
    for turn, sizes in enumerate(([5, 1, 2, 23], [1, 1, 17, 2], [40, 3, 1])):
        cut = {r: portions(length[r], sizes[i % len(sizes):] + sizes) for i, r in enumerate(names)}
        while any(cut.values()):
            step = [(r, cut[r].pop(0)) for j, r in enumerate(names) if cut[r] and (len(mixed) + j + turn) % 4]
            if step:
                mixed.append(step)
            else:
                mixed.append([(r, cut[r].pop(0)) for r in names if cut[r]])
    out["mixed"] = mixed
    return out


# ---- one op through a runtime -----------------------------------------------------------------------------
def run_op(op, args, gpu: bool, vars_=None):
    """Execute one op: `args` in interface order — tensors (states: uint8), or numbers. Returns the tensors afterwards."""
    vars_ = vars_ or {}
    doc = {"schema_version": 7, "model": "one-op", "vars": {n: {"max": v} for n, v in vars_.items()}, "states": {}, "buffers": {},
           "ops": {"op": op}, "programs": {"go": {"calls": [{"op": "op", "args": []}]}},
           "modules": {}}
    used = {l["module"] for l in op["impl"]["launches"]}
    doc["modules"] = {n: m for n, m in C.modules_for(sorted(used)).items() if n in used}
    call, names = doc["programs"]["go"]["calls"][0]["args"], []
    for i, (a, p) in enumerate(zip(args, op["params"])):
        name = f"b{i}"
        if not isinstance(a, torch.Tensor):
            call.append({p: a})
        elif p.endswith("state"):
            doc["states"][name] = {"bytes": a.numel()}
            call.append({"state": name})
            names.append((i, name))
        else:
            doc["buffers"][name] = {"dtype": p[p.index("<") + 1:-1], "shape": [max(1, a.numel())], "kind": "inout"}
            call.append({"buf": name})
            names.append((i, name))
    assert len(args) == len(op["params"])
    # a var the op's launches do not read may not be declared
    import json
    text = json.dumps(op)
    doc["vars"] = {n: v for n, v in doc["vars"].items() if f'"{n}"' in text}
    if gpu:
        from kern_b200.runtime import Runtime

        rt = Runtime(doc, guard_bands=True)
    else:
        from kern_b200.cpu import CpuRuntime

        rt = CpuRuntime(doc)
    for i, name in names:
        rt.tensor(name).view(-1)[: args[i].numel()].copy_(args[i].reshape(-1))
    if gpu:
        torch.cuda.synchronize()
    rt.issue("go", vars_)
    rt.synchronize()
    out = {i: rt.tensor(name).view(-1)[: args[i].numel()].cpu().clone().view(args[i].shape) for i, name in names}
    if gpu:
        assert rt.check_guards() == []
    return out

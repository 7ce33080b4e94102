"""Prefill and decode throughput of a decoder with listed layers beside the framework's closest model at equal size, with the
time of every kind of kernel against its roofline: `python bench.py --config gafapel|barotar|diderax|fusasun [--layers N]`.

The decoders have the width, depth, vocabulary and routed experts of the 48B-A3B shape class and random weights. Gafapel has
Mamba-2 and unrotated latent-attention layers over four residual streams, Barotar window attention beside time mixing and gated
linear attention, Diderax gated linear attention, grouped-query attention and 512 + 64 latent attention with sinks; the model beside
them per-key-decay delta-rule layers and 512 + 64 latent attention. Beside Barotar and Diderax there is also the routed decoder
with grouped-query attention of the same head counts and dims, for its attention kernels. Fusasun has window attention beside
pooled blocks and 512 + 64 latent attention in a window; beside it Diderax, and Barotar for its window attention. A point is timed end to end (CUDA events around the call, captured graphs for decode,
L2 flushed before every sample) and once more call by call, where a call's roofline is the larger of its bytes over the
measured copy rate and its flops over the measured tensor rate.
"""
from __future__ import annotations

import json
import re
from pathlib import Path

MODELS = {"gafapel": ("gafapel-48b-a3b", "latent-48b-a3b"), "barotar": ("barotar-48b-a3b", "latent-48b-a3b", "moe-30b-a3b"),
          "diderax": ("diderax-48b-a3b", "latent-48b-a3b", "moe-30b-a3b"), "fusasun": ("fusasun-48b-a3b", "diderax-48b-a3b", "barotar-48b-a3b")}
POINTS = ({"groups": 1, "chunk": 2048, "context": 2048}, {"groups": 4, "chunk": 512, "context": 2048},
          {"groups": 1, "rows": 1, "context": 1024}, {"groups": 16, "rows": 1, "context": 1024}, {"groups": 64, "rows": 1, "context": 1024})


def peaks() -> tuple[float, float, str]:
    p = Path(__file__).resolve().parent.parent.parent / "MEASURED_PEAKS.json"
    if p.exists():
        d = json.loads(p.read_text())
        if "hbm_gbs" in d and "bf16_tflops" in d:
            return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def cost(doc: dict, call: dict, groups: int, rows: int, context: int) -> tuple[float, float]:
    """(bytes, flops) a call must at least move and do: weights once (routed experts: those the tokens can reach), every
    token-shaped argument once, the states it reads and writes, and the products it is made of."""
    op, n = call["op"], groups * rows
    seen, bufs = set(), []
    for a in call["args"]:                                  # columns of one buffer bound several times are read once
        if "buf" in a and a["buf"] not in seen and not a["buf"].startswith("rope."):
            seen.add(a["buf"])
            b = doc["buffers"][a["buf"]]
            derived = b["kind"] == "carry" and isinstance(b["shape"][0], int) and b["dtype"] == "bf16"      # weights put together at load
            bufs.append((a, b | {"kind": "weight"} if derived else b))
    es = {"bf16": 2, "f32": 4, "i32": 4, "i64": 8}
    wbytes = sum(2 * _prod(b["shape"]) for _, b in bufs if b["kind"] == "weight")
    w = [b["shape"] for _, b in bufs if b["kind"] == "weight"]
    tok = 0.0
    for _, b in bufs:
        if b["kind"] != "weight" and b["shape"][0] == "tokens":
            tok += n * es.get(b["dtype"], 4) * _prod(b["shape"][1:])
        elif b["kind"] != "weight" and b["shape"][0] == "seqs":
            tok += groups * es.get(b["dtype"], 4) * _prod(b["shape"][1:])
    flops = 0.0
    st = [doc["states"][a["state"]] for a in call["args"] if "state" in a]
    for s in st:
        if s.get("bytes_per_seq"):
            tok += 2 * groups * s["bytes_per_seq"]
    m = re.match(r"latent_attn_[pd]_(\d+)x(\d+)x(\d+)x\d+n?(?:w(\d+))?", op)
    if m:                                                   # heads, latent columns, rotated columns behind them, window
        H, rank, rot = map(int, m.groups()[:3])
        window = int(m.group(4) or 1 << 30)
        flops = 2.0 * groups * H * (2 * rank + rot) * sum(min(p + 1, window) for p in range(context - rows, context))
        return n * H * (2 * rank + rot) * 2.0 + groups * min(context, window + rows - 1) * (rank + rot) * 2.0, flops
    if op.startswith("moe_table_"):                         # a row of the table, an expert and a weight per choice
        return n * (8 + 12.0 * int(op.rsplit("x", 1)[1])), 0.0
    m = re.match(r"prep_pool_[pd]_(\d+)x(\d+)x(\d+)x(\d+)x\d+x(\d+)x", op)
    if m:                                                   # q read and written, keys and values read, written and read for their means
        hq, hk, d, dv, pool = map(int, m.groups())
        return n * 2.0 * (2 * hq * d + hk * (d + dv) * (3 + 1 / pool)), 0.0
    m = re.match(r"pooled_attn_[pd]_(\d+)x(\d+)x(\d+)x(\d+)x(\d+)x(\d+)x", op)
    if m:
        hq, hk, d, dv, window, pool = map(int, m.groups())
        seen_by = lambda p: min(p + 1, window) + max(0, p - window + 1) // pool
        flops = 2.0 * groups * hq * (d + dv) * sum(seen_by(p) for p in range(context - rows, context))
        keys = min(context, window + rows - 1) + max(0, context - window) // pool
        return n * hq * (d + dv) * 2.0 + groups * keys * hk * (d + dv) * 2.0, flops
    m = re.match(r"prep_whole_(\d+)x(\d+)x(\d+)x", op)
    if m:                                                   # q read and written, k read, keys and values written
        hq, hk, d = map(int, m.groups())
        return n * (2 * hq + 3 * hk) * d * 2.0, 0.0
    if re.match(r"(window_|sink_)?attn_(prefill|decode|p_|d_)", op):
        hq, hk, d, dv, window = _heads(doc, call)
        seen_by = lambda p: min(p + 1, window)
        flops = 2.0 * groups * hq * (d + dv) * sum(seen_by(p) for p in range(context - rows, context))
        cols = groups * rows * (hq * (d + dv + (dv if op.startswith("sink_") else 0))) * 2.0      # with the gate's columns
        return cols + groups * min(context, window + rows - 1) * hk * (d + dv) * 2.0, flops
    m = re.match(r"lin_[pd]_(\d+)x(\d+)x(\d+)", op)
    if m:                                                   # a recurrence: its rows, its decays and its states
        H, dk, dv = map(int, m.groups())
        return n * H * (2 * dk + 3 * dv) * 2.0 + n * H * dk * 4.0 + 2.0 * groups * H * dk * dv * 4, 0.0
    if op.startswith("shift_"):
        width, targets = doc["buffers"][call["args"][1]["buf"]]["shape"][::-1]
        return (n * (1 + targets) + targets) * width * 2.0 + 2.0 * groups * width * 4, 0.0
    m = re.search(r"_(\d+)x(\d+)_of\d+$", op)
    if m:                                                   # columns of wider rows
        a, b = map(int, m.groups())
        return a * b * 2.0 + n * (2.0 * b + 4.0 * a), 2.0 * n * a * b
    if "moe_fc" in op:
        E, a, b = w[0]
        k = next(x for _, x in bufs if x["shape"][0] == "tokens")["shape"]
        top = k[1] if len(k) == 3 else doc["buffers"]["moe.ids"]["shape"][1]
        hit = E * (1 - (1 - top / E) ** n)
        wbytes = wbytes * hit / E
        flops = 2.0 * n * top * a * b
    elif w and len(w[0]) == 3:
        flops = 2.0 * n * _prod(w[0])
    elif w and len(w[0]) == 2 and op.split("_")[0] in ("lin", "glu", "geglu", "qkv", "head", "router", "q", "v", "qa", "o", "kda", "gate", "down", "lm", "moe"):
        mats = [x for x in w if len(x) == 2]
        m = groups if doc["buffers"][call["args"][0]["buf"]]["shape"][0] == "seqs" else n
        flops = sum(2.0 * m * _prod(x) for x in mats)
        if op == "embed":
            flops = 0.0
    elif op.startswith("embed"):
        wbytes = n * 4 * w[0][1]
    elif "attn" in op and st:
        per = st[0]["bytes_per_token"] / 2                      # columns of a cached row
        reach = context if rows == 1 else context - (rows - 1) / 2
        heads = _prod([doc["buffers"][call["args"][0]["buf"]]["shape"][1]]) / per
        tok += groups * context * per * 2
        flops = 4.0 * n * heads * per * reach
    if op.startswith("embed_"):
        wbytes = n * 2 * w[0][1]
    elif op == "embed":
        wbytes = n * 4 * doc["buffers"][call["args"][7]["buf"]]["shape"][1] if len(call["args"]) > 7 else n * 2 * w[0][1]
    return wbytes + tok, flops


def _heads(doc: dict, call: dict) -> tuple[int, int, int, int, int]:
    """(query heads, key heads, key columns, value columns, window) of a grouped-query attention call."""
    m = re.match(r"window_attn_._(\d+)x(\d+)x(\d+)x(\d+)x(\d+)", call["op"])
    if m:
        return tuple(map(int, m.groups()))
    m = re.match(r"sink_attn_._(\d+)x(\d+)x(\d+)x", call["op"])
    if m:
        hq, hk, d = map(int, m.groups())
        return hq, hk, d, d, 1 << 30
    args = doc["ops"][call["op"]]["impl"]["launches"][0]
    d = int(re.search(r"_d(\d+)", args["entry"]).group(1))
    hk = doc["states"][next(a["state"] for a in call["args"] if "state" in a)]["bytes_per_token"] // (4 * d)
    return doc["buffers"][call["args"][2]["buf"]]["shape"][1] // d, hk, d, d, 1 << 30


def _prod(v) -> float:
    out = 1.0
    for x in v:
        out *= x
    return out


def run(model: str, layers: int, points, samples: int, by_call: bool = True) -> list[dict]:
    import numpy as np
    import torch

    from ..cli import bench_points
    from ..engine import Engine
    from ..models import registry
    from ..runtime import Runtime

    hbm, tflops, _ = peaks()
    cfg, build, load, _ = registry.resolve(model, layers=layers, max_tokens=2048, max_seqs=64, max_context=4096)
    rt = Runtime(build(cfg), tokens=64 * 1088 + 4096, slots=132)
    load(rt, cfg)
    rt.once()
    out = []
    for pt, r in zip(points, bench_points(rt, {"samples": samples, "seed": 0, "sweep": list(points)}, quiet=True)["points"]):
        g, rows, ctx = r["groups"], r["rows"], r["context"]
        rec = {"model": model, "layers": layers, "groups": g, "rows": rows, "context": ctx, "ms": round(r["p50_ms"], 4),
               "tok_s": round(g * rows / r["p50_ms"] * 1e3, 1)}
        if by_call:
            eng, rng = Engine(rt), np.random.default_rng(1)
            seqs = [eng.open(ctx) for _ in range(g)]
            for i in range(0, ctx - rows, 2048 // g):
                eng.step([(s, rng.integers(1, 200, min(2048 // g, ctx - rows - i)).tolist()) for s in seqs])
            best = None
            for _ in range(5):
                eng.step([(s, rng.integers(1, 200, rows).tolist()) for s in seqs], timed=True)
                for s in seqs:
                    s.length -= rows
                    del s.tokens[-rows:]
                t = [x[2] for x in eng.last_times]
                best = t if best is None else [min(a, b) for a, b in zip(best, t)]
            calls = rt.doc["programs"]["prefill" if rows > 1 else "decode"]["calls"]
            ops: dict[str, list] = {}
            for c, ms in zip(calls, best):
                nbytes, flops = cost(rt.doc, c, g, rows, ctx)
                e = ops.setdefault(c["op"], [0.0, 0.0, 0])
                e[0] += ms; e[1] += max(nbytes / hbm, flops / tflops) * 1e3; e[2] += 1
            rec["by_op"] = {o: {"calls": n, "ms": round(ms / n, 4), "roofline_ms": round(roof / n, 4), "times_roofline": round(ms / max(roof, 1e-9), 1)}
                            for o, (ms, roof, n) in sorted(ops.items(), key=lambda kv: -kv[1][0])}
            for s in seqs:
                eng.close(s)
        out.append(rec)
    del rt
    torch.cuda.empty_cache()
    return out


def main(args) -> int:
    layers = args.layers if args.layers != 36 else 8
    hbm, tf, src = peaks()
    for model in MODELS[args.config]:
        for rec in run(model, layers, POINTS, max(12, min(args.steps, 24))):
            rec["peaks"] = {"copy_tb_s": round(hbm / 1e12, 2), "bf16_pflop_s": round(tf / 1e15, 2), "source": src}
            rec["data"] = "synthetic (random-init weights, random token ids)"
            print(json.dumps(rec), flush=True)
    return 0

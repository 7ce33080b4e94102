"""Op builders of the decoder blocks that take any size and either activation type (bf16, or f32 in a model's 32-bit
form): matrix products, hyper-connections, the residual with norms on both sides, the Mamba-2 mixer, linear attention with a
decay per key channel, latent attention with or without rotated columns, attention in a sliding window, beside pooled blocks, or
with a sink and an output gate, a convolution added to its input, routed experts. Where a bf16 size fits the tensor-core kernels the op is the one `common.py` builds or the
tensor-core form of the mechanism; the rest runs generic kernels. Weights are bf16 in both forms.
"""
from __future__ import annotations

from . import common as C

ACT_BYTES = {"bf16": 2, "f32": 4}


def _launch(module: str, entry: str, block, grid, lp, args, **kw) -> dict:
    return {"module": module, "entry": entry, "block": block, "grid": grid, "params": lp, "args": args, **kw}


def _op(iface, *launches, **impl) -> dict:
    return {"params": iface, "impl": {"launches": list(launches), **impl}}


P = lambda i: {"param": i}
I = lambda v: {"i32": v}
L = lambda v: {"i64": v}
NULL = ("i64", {"i64": 0})


def chain_ops(*ops, inner: dict | None = None, scratch: dict | None = None) -> dict:
    """Ops one after the other as one op (one call of a program): the interfaces in order, without the params that `inner` —
    {(op, param): scratch name} — ties together through `scratch`."""
    inner, iface, launches, room = inner or {}, [], [], dict(scratch or {})
    for n, o in enumerate(ops):
        at = {}
        for i, t in enumerate(o["params"]):
            if (n, i) not in inner:
                at[i] = len(iface)
                iface.append(t)

        def sub(x):
            if isinstance(x, list):
                return [sub(v) for v in x]
            if not isinstance(x, dict):
                return x
            if set(x) == {"param"} and (n, x["param"]) in inner:
                return {"scratch": inner[n, x["param"]]}
            if set(x) == {"scratch"}:
                return {"scratch": f"{n}.{x['scratch']}"}
            return {k: at[v] if k == "param" else (v if k == "when" else sub(v)) for k, v in x.items()}

        launches += [sub(l) | {"params": l["params"]} for l in o["impl"]["launches"]]
        room |= {f"{n}.{k}": v for k, v in o["impl"].get("scratch", {}).items()}
    return _op(iface, *launches, **({"scratch": room} if room else {}))


def tiles_fit(*extents: int) -> bool:
    """Whether rows of these lengths are whole 16-byte vectors of bf16, which the tensor-core tiles and TMA need."""
    return all(e % 8 == 0 for e in extents)


# ---- matrix products ----------------------------------------------------------------------------------
def _generic(sfx: str, iface, n: int, k: int, lda: int, ldc: int, rows_var: str, batch: int = 1, w=None, strides=(0, 0, 0),
             limit: float = 0.0, bias=NULL) -> dict:
    """`w`: (row stride, column stride) of the weights in elements; `strides`: what a step of the batch adds to A, W, C."""
    wsn, wsk = w or (k, 1)
    return _launch("linear", f"kern_linear_{sfx}", [256, 1, 1], [-(-n // 64), {"ceil_div": [rows_var, 64]}, batch],
                   iface[:3] + ["i32"] * 5 + ["i64"] * 5 + ["out buffer<i32>", "f32", bias[0]],
                   [P(0), P(1), P(2), P(3), I(n), I(k), I(lda), I(ldc), L(wsn), L(wsk), *map(L, strides), P(4), {"f32": limit}, bias[1]])


GLUS = ("swiglu", "geglu", "clamped")      # gated units over [gate rows ; up rows]; `clamped` takes a limit


def linear_op(n: int, k: int, *, act: str = "bf16", epilogue: str = "store", rows_var: str = "tokens", rows_max: int,
              lda: int | None = None, ldc: int | None = None, limit: float = 0.0, bias: bool = False) -> dict:
    """C[rows, n] = A[rows, k] . W[n, k]^T. Interface [a, w, c, rows, err]; epilogue store | f32 | a gated unit as in `gemm_op`.
    `bias` (swiglu): one per row of W, at the end of the interface."""
    if bias and epilogue != "swiglu":
        raise ValueError(f"biases in a product with epilogue `{epilogue}`")
    lda = k if lda is None else lda
    cols = n // 2 if epilogue in GLUS else n
    ldc = cols if ldc is None else ldc
    if act == "bf16" and epilogue != "clamped" and tiles_fit(cols, k, lda, ldc):
        return C.gemm_op(n, k, epilogue=epilogue + ("_bias" if bias else ""), rows_var=rows_var, rows_max=rows_max, lda=lda, ldc=ldc)
    out = "f32" if epilogue == "f32" else act
    sfx = act + {"store": "", "f32": "_f32" if act == "bf16" else ""}.get(epilogue, "_" + epilogue)
    iface = [f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{out}>", "i32", "out buffer<i32>"] + (["in buffer<bf16>"] if bias else [])
    return _op(iface, _generic(sfx, iface, cols, k, lda, ldc, rows_var, limit=limit, bias=(iface[5], P(5)) if bias else NULL))


def head_tiles(n: int, k: int, lda: int, ldc: int, act: str) -> bool:
    """Whether per-head products of this size run on the tensor-core tiles (which read weights as [n, k])."""
    return act == "bf16" and tiles_fit(n, k, lda, ldc)


def head_linear_op(heads: int, n: int, k: int, *, act: str = "bf16", rows_max: int, lda: int, ldc: int, transposed: bool = False) -> dict:
    """Per head h: C[:, h n : (h + 1) n] = A[:, h k : (h + 1) k] . W_h^T, with W_h [n, k] stacked by head, or [k, n] when
    `transposed`. Interface [a, w, c, rows, err]."""
    iface = [f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{act}>", "i32", "out buffer<i32>"]
    if head_tiles(n, k, lda, ldc, act) and not transposed:
        tmap = lambda param, dims, strides, box: {"pack": {"size": 128, "fields": [{"at": 0, "tensormap": {
            "param": param, "dtype": "bf16", "dims": dims, "strides": strides, "box": box, "swizzle": 128, "l2_promotion": 256}}]}}
        launches = []
        # wide tiles once they give every SM one
        wide = [(256, 4 * C.BM + 1, rows_max), (128, 1, min(4 * C.BM, rows_max))] if n >= 256 else [(128 if n >= 128 else 64, 1, rows_max)]
        for bn, lo, hi in wide:
            if lo > hi:
                continue
            when = {"var": "tokens", **({"min": lo} if lo > 1 else {}), **({"max": hi} if hi < rows_max else {})}
            launches.append(_launch(
                "gemm_bf16", f"kern_gemm_bf16_heads_n{bn}", [192, 1, 1], [C.SMS, 1, 1],
                ["bytes<128>", "bytes<128>", iface[2]] + ["i32"] * 5 + ["out buffer<i32>"],
                [tmap(0, [heads * k, 0], [lda * 2], [C.BK, C.BM]), tmap(1, [k, n, heads], [k * 2, n * k * 2], [C.BK, bn, 1]),
                 P(2), P(3), I(n), I(k), I(ldc), I(heads), P(4)], shared_mem=C.gemm_smem(bn), **({"when": when} if len(when) > 1 else {})))
        return _op(iface, *launches)
    return _op(iface, _generic(act, iface, n, k, lda, ldc, "tokens", heads, (1, n) if transposed else (k, 1), (k, n * k, n)))


def gate_mul_op(d: int, gate_stride: int, act: str = "bf16") -> dict:
    """out = x * sigmoid(gate). Interface [x, gate, out, tokens]."""
    iface = [f"in buffer<{act}>", f"in buffer<{act}>", f"out buffer<{act}>", "i32"]
    return _op(iface, _launch("linear", f"kern_gate_mul_{act}", [256, 1, 1], [-(-d // 1024), {"clamp": ["tokens", 0, 4096]}, 1],
                              iface + ["i32"] * 4, [P(0), P(1), P(2), P(3), I(d), I(d), I(gate_stride), I(d)]))


def transpose_heads_op(heads: int, rows: int, cols: int) -> dict:
    """[heads][rows][cols] -> [heads][cols][rows]. Interface [src, dst]."""
    iface = ["in buffer<bf16>", "out buffer<bf16>"]
    return _op(iface, _launch("linear", "kern_transpose_heads_bf16", [256, 1, 1], [-(-cols // 32), -(-rows // 32), heads],
                              iface + ["i32", "i32"], [P(0), P(1), I(rows), I(cols)]))


def copy_cols_op(rows: int, cols: int, stride: int) -> dict:
    """A [rows, cols] matrix into columns of one whose rows are `stride` wide. Interface [src, dst]."""
    iface = ["in buffer<bf16>", "inout buffer<bf16>"]
    return _op(iface, _launch("linear", "kern_copy_cols_bf16", [256, 1, 1], [rows, 1, 1], iface + ["i32", "i32"], [P(0), P(1), I(cols), I(stride)]))


# ---- hyper-connections ----------------------------------------------------------------------------------
HYPER_COUNTS = (1, 2, 3, 4)      # stream counts with a kernel of their own
HYPER_MAX = 16


def _hyper_entry(kind: str, act: str, streams: int) -> str:
    if not 1 <= streams <= HYPER_MAX:
        raise ValueError(f"{streams} residual streams: 1 to {HYPER_MAX} are supported")
    return f"kern_hyper_{kind}_{act}_s{streams if streams in HYPER_COUNTS else 0}"


def hyper_embed_op(width: int, streams: int, vocab: int, max_pos: int, eps: float, act: str = "bf16") -> dict:
    """Token row + position row, RMS norm, into every stream, and the first sublayer's normed input.
    Interface [ids, positions, table, position table, norm w, stream weights in, next norm w, x, xn, err]."""
    iface = ["in buffer<i64>", "in buffer<i64>"] + ["in buffer<bf16>"] * 5 + ["out buffer<f32>", f"out buffer<{act}>", "out buffer<i32>"]
    return _op(iface, _launch("hyper", f"kern_hyper_embed_{act}", [256, 1, 1], ["tokens", 1, 1],
                              iface[:9] + ["i32"] * 4 + ["f32", "out buffer<i32>"],
                              [*map(P, range(9)), I(width), I(streams), I(vocab), I(max_pos), {"f32": eps}, P(9)], shared_mem=width * 4))


def hyper_mix_op(width: int, streams: int, eps: float, act: str = "bf16", routed: int = 0) -> dict:
    """A sublayer's result into the streams, and the next sublayer's normed input.
    Interface [x, y, mix, out, next in, next norm w, xn], with `routed` (experts per token) also [perm, weights] at the end:
    y then holds expert-sorted rows and a token's result is the weighted sum of its own."""
    iface = ["inout buffer<f32>", f"in buffer<{act}>"] + ["in buffer<bf16>"] * 4 + [f"out buffer<{act}>"]
    iface += ["in buffer<i32>", "in buffer<f32>"] if routed else []
    pt, pa = (iface[7:9], [P(7), P(8)]) if routed else ([NULL[0]] * 2, [NULL[1]] * 2)
    return _op(iface, _launch("hyper", _hyper_entry("mix", act, streams), [256, 1, 1], ["tokens", 1, 1],
                              iface[:2] + pt + iface[2:7] + ["i32", "i32", "i32", "f32"],
                              [P(0), P(1), *pa, *map(P, range(2, 7)), I(width), I(streams), I(routed), {"f32": eps}], shared_mem=width * 4))


def hyper_last_op(width: int, streams: int, act: str = "bf16", routed: int = 0) -> dict:
    """The last sublayer: the sum of the new streams. Interface [x, y, mix, out, hidden] (+ [perm, weights])."""
    iface = ["in buffer<f32>", f"in buffer<{act}>", "in buffer<bf16>", "in buffer<bf16>", "out buffer<f32>"]
    iface += ["in buffer<i32>", "in buffer<f32>"] if routed else []
    pt, pa = (iface[5:7], [P(5), P(6)]) if routed else ([NULL[0]] * 2, [NULL[1]] * 2)
    return _op(iface, _launch("hyper", _hyper_entry("last", act, streams), [256, 1, 1], ["tokens", 1, 1],
                              iface[:2] + pt + iface[2:5] + ["i32", "i32", "i32"],
                              [P(0), P(1), *pa, P(2), P(3), P(4), I(width), I(streams), I(routed)]))


def row_norm_op(width: int, eps: float, src_rows: int, act: str = "bf16", pick: str = "each") -> dict:
    """RMS norm of f32 rows: `each` of a one-row-per-sequence call's rows, the `last` row of every sequence of a ragged call, or the
    rows a list names (`listed`, over var `wanted`). Interface [src, w, y] (+ [cu_seqlens] or [rows])."""
    iface = ["in buffer<f32>", "in buffer<bf16>", f"out buffer<{act}>"] + ([] if pick == "each" else ["in buffer<i32>"])
    p3 = ("in buffer<i32>", P(3))
    cu, rows = (p3 if pick == "last" else NULL), (p3 if pick == "listed" else NULL)
    return _op(iface, _launch("hyper", f"kern_row_norm_f32_{act}", [256, 1, 1], ["wanted" if pick == "listed" else "seqs", 1, 1],
                              [iface[0], cu[0], rows[0], iface[1], iface[2], "i32", "i32", "f32"],
                              [P(0), cu[1], rows[1], P(1), P(2), I(src_rows), I(width), {"f32": eps}], shared_mem=width * 4))


# ---- Mamba-2 (state-space duality) ----------------------------------------------------------------------
def ssd_line_bytes(heads: int, vdim: int, state: int, channels: int, taps: int, act: str = "bf16") -> tuple[int, int]:
    """(bytes of one per-sequence line, offset of the recurrent matrix in it)."""
    s_off = ((taps - 1) * channels * ACT_BYTES[act] + 255) // 256 * 256
    return (s_off + heads * vdim * state * 4 + 255) // 256 * 256, s_off


def short_conv_op(channels: int, taps: int, x_stride: int, line_bytes: int, ragged: bool, act: str = "bf16", x_off: int = 0) -> dict:
    """Causal convolution with bias, then SiLU, for any taps / channels; the window at the start of the state line
    advances with it. `x_off`: elements before the channels in a row (decides whether the aligned kernels apply).
    Interface [x, y, state, lines, (cu_seqlens,) w, bias, seqs, rows]."""
    if act == "bf16" and 2 <= taps <= 4 and channels % 4 == 0 and x_stride % 4 == 0 and x_off % 4 == 0:
        return C.gdn_conv_op(channels, taps, x_stride, line_bytes, ragged, bias=True)
    iface = [f"in buffer<{act}>", f"out buffer<{act}>", "inout state", "in buffer<i32>"] + (["in buffer<i32>"] if ragged else [])
    w = len(iface)
    iface += ["in buffer<bf16>", "in buffer<bf16>", "i32", "i32"]
    cu_t, cu_a = ("in buffer<i32>", P(4)) if ragged else NULL
    cols = -(-channels // 256)
    conv = _launch("ssd", f"kern_ssd_conv_{act}", [256, 1, 1], ["tokens", cols, 1],
                   [iface[0], iface[1], "in state", "in buffer<i32>", cu_t, "in buffer<bf16>", "in buffer<bf16>"] + ["i32"] * 5 + ["i64"],
                   [P(0), P(1), P(2), P(3), cu_a, P(w), P(w + 1), P(w + 2), P(w + 3), I(channels), I(taps), I(x_stride), L(line_bytes)])
    upd = _launch("ssd", f"kern_ssd_conv_state_{act}", [256, 1, 1], ["seqs", cols, 1],
                  [iface[0], "inout state", "in buffer<i32>", cu_t] + ["i32"] * 4 + ["i64"],
                  [P(0), P(2), P(3), cu_a, P(w + 2), I(channels), I(taps), I(x_stride), L(line_bytes)])
    return _op(iface, conv, upd)


SSD_CHUNK_MIN = 8       # rows of a call from which a sequence is computed in chunks


def ssd_rule_op(heads: int, vdim: int, state: int, groups: int, dt_stride: int, line_bytes: int, s_off: int, ragged: bool,
                act: str = "bf16") -> dict:
    """The recurrence. Interface [xbc, dt, y (f32), state, lines, (cu_seqlens,) A_log, dt_bias, D, seqs]."""
    if heads % groups or state > 512:
        raise ValueError(f"{heads} heads in {groups} groups with {state} state columns: heads split evenly, at most 512 columns")
    iface = [f"in buffer<{act}>", f"in buffer<{act}>", "out buffer<f32>", "inout state", "in buffer<i32>"] + (["in buffer<i32>"] if ragged else [])
    w = len(iface)
    iface += ["in buffer<bf16>"] * 3 + ["i32"]
    cu_t, cu_a = ("in buffer<i32>", P(5)) if ragged else NULL
    nl = next(n for n in (32, 64, 128, 256, 512) if state <= n)
    lp = iface[:5] + [cu_t] + ["in buffer<bf16>"] * 3 + ["i32"] * 6 + ["i64", "i32"]
    args = [*map(P, range(5)), cu_a, *map(P, range(w, w + 4)), I(heads), I(vdim), I(state), I(groups), I(dt_stride), L(line_bytes), I(s_off)]
    chunked = ragged and act == "bf16" and state <= 256
    tb = (32 if nl <= 128 else 8) if ragged and not chunked else (SSD_CHUNK_MIN if chunked else 1)
    rule = _launch("ssd", f"kern_ssd_rule_{act}_n{nl}", [256, 1, 1], [heads * -(-vdim // 16), "seqs", 1], lp + ["i32", "i32"],
                   args + [I(tb), I(SSD_CHUNK_MIN - 1 if chunked else C.I32_MAX)], shared_mem=tb * (2 * state + 16 + 2) * 4)
    if not chunked:
        return _op(iface, rule)
    # a ragged call's long sequences in chunks on the tensor cores, its few-row ones (decode rows among prompts) row by row
    np_, q = nl, 64
    smem = 2 * (2 * q * (np_ + 8) + q * 40) * 2 + 3 * 32 * (np_ + 8) * 2 + q * 32 * 4 + 5 * q * 4
    chunk = _launch("ssd_chunk", f"kern_ssd_chunk_n{np_}", [256, 1, 1], [heads * -(-vdim // 32), "seqs", 1], lp + ["i32"],
                    args + [I(SSD_CHUNK_MIN)], shared_mem=smem)
    return _op(iface, chunk, rule)


def ssd_gate_norm_op(inner: int, parts: int, z_stride: int, eps: float, act: str = "bf16") -> dict:
    """out = rms_norm per part of (y * silu(z)), times w. Interface [y (f32), z, w, out]."""
    if inner % parts:
        raise ValueError(f"{inner} columns do not split into {parts} norm groups")
    iface = ["in buffer<f32>", f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{act}>"]
    return _op(iface, _launch("ssd", f"kern_ssd_gate_norm_{act}", [min(256, -(-inner // parts // 128) * 32), 1, 1], ["tokens", parts, 1], iface + ["i32", "i32", "i32", "f32"],
                              [*map(P, range(4)), I(inner), I(parts), I(z_stride), {"f32": eps}], shared_mem=inner // parts * 4))


# ---- latent attention without positions -----------------------------------------------------------------
def latent_append_op(rank: int, stride: int, eps: float, act: str = "bf16") -> dict:
    """RMS norm of a token's latent into its row of the paged cache. Interface [latent columns, state, slots, norm w]."""
    iface = [f"in buffer<{act}>", "inout state", "in buffer<i64>", "in buffer<bf16>"]
    return _op(iface, _launch("latent", f"kern_latent_append_{act}", [128, 1, 1], ["tokens", 1, 1], iface + ["i32", "i32", "f32"],
                              [*map(P, range(4)), I(rank), I(stride), {"f32": eps}]))


def latent_attn_op(heads: int, rank: int, scale: float, page_size: int, table_width: int, ragged: bool, act: str = "bf16",
                   seqs_max: int = 0) -> dict:
    """Every head attends over the shared latent rows, which are keys and values alike.
    Interface [q, state, out, block_table, lens, err] (+ [row_seq] for ragged rows: one attention row per token). bf16
    latents of up to 512 aligned columns take the tensor-core kernel, others one block per (row, head)."""
    if act == "bf16" and tiles_fit(rank) and rank <= 512 and (page_size % 64 == 0 or 64 % page_size == 0):
        return C.mla_attn_op(heads, page_size, table_width, ragged, seqs_max=seqs_max, rank=rank, scale=scale)
    if rank > 1024:
        raise ValueError(f"latent rows of {rank} columns (at most 1024)")
    iface = [f"in buffer<{act}>", "in state", f"out buffer<{act}>", "in buffer<i32>", "in buffer<i32>", "out buffer<i32>"]
    iface += ["in buffer<i32>"] if ragged else []
    w = next(n for n in (64, 128, 256, 512, 1024) if rank <= n)
    return _op(iface, _launch("latent", f"kern_latent_attn_{act}_w{w}", [128, 1, 1], [heads, "tokens" if ragged else "seqs", 1],
                              iface[:5] + ["in buffer<i32>" if ragged else "i64", "i32", "i32", "i32", "i32", "f32", "out buffer<i32>"],
                              [*map(P, range(5)), P(6) if ragged else NULL[1], I(heads), I(rank), I(table_width), I(page_size),
                               {"f32": scale}, P(5)], shared_mem=(4 * rank + 8) * 4))


# ---- latent attention with a rotated part: sinks, windows, gates ------------------------------------------------------------
def latent_prep_op(rank: int, rot: int, q_rank: int, stride: int, q_stride: int, max_pos: int, eps: float, act: str = "bf16", halves: bool = True) -> dict:
    """Of a projected row [query latent | latent | rotated key part]: the query latent normed into rows of its own, the latent
    normed and the key part turned (pairs i, i + rot / 2, or neighbours) into a row of the paged cache.
    Interface [rows, state, q latent, positions, slots, cos, sin, latent norm w, query norm w, err]."""
    if rot % 2 or not rot:
        raise ValueError(f"a rotated key part of {rot} columns")
    if rank + q_rank > 50000:
        raise ValueError(f"latents of {rank} and {q_rank} columns (at most 50000 together)")
    iface = [f"in buffer<{act}>", "inout state", f"out buffer<{act}>", "in buffer<i64>", "in buffer<i64>", "in buffer<f32>", "in buffer<f32>", "in buffer<bf16>",
             "in buffer<bf16>", "out buffer<i32>"]
    return _op(iface, _launch("latent", f"kern_latent_prep_{act}", [256, 1, 1], ["tokens", 1, 1], iface[:9] + ["i32"] * 7 + ["f32", "out buffer<i32>"],
                              [*map(P, range(9)), I(rank), I(rot), I(int(halves)), I(q_rank), I(stride), I(q_stride), I(max_pos), {"f32": eps}, P(9)], shared_mem=(rank + q_rank) * 4))


def latent_rot_attn_op(heads: int, rank: int, rot: int, scale: float, page_size: int, table_width: int, max_pos: int, rot_stride: int, ragged: bool,
                       act: str = "bf16", seqs_max: int = 0, *, sink: bool = True, halves: bool = True, window: int = C.I32_MAX, gate_stride: int = 0) -> dict:
    """`latent_attn_op` over rows with `rot` rotated key columns behind the latent, with a sink per head, over the last `window`
    positions, the result times sigmoid of a gate per head (`gate_stride`: the row stride of the gates; sinks and gates not both).
    Interface [q, state, out, block_table, lens, err] (+ [row_seq] for ragged rows), then [q_rot, cos, sin], [sink], [gate]."""
    if act == "bf16" and tiles_fit(rank, rot) and rank <= 512 and rot <= 64 and (page_size % 64 == 0 or 64 % page_size == 0):
        return C.mla_attn_op(heads, page_size, table_width, ragged, seqs_max=seqs_max, rank=rank, scale=scale, rot=rot, max_pos=max_pos, rot_stride=rot_stride,
                             sink=sink, halves=halves, window=window, gate_stride=gate_stride)
    if rank > 1024:
        raise ValueError(f"latent rows of {rank} columns (at most 1024)")
    iface = [f"in buffer<{act}>", "in state", f"out buffer<{act}>", "in buffer<i32>", "in buffer<i32>", "out buffer<i32>"]
    iface += ["in buffer<i32>"] if ragged else []
    o = len(iface)
    iface += [f"in buffer<{act}>", "in buffer<f32>", "in buffer<f32>"]
    extra, more = C.latent_extra(iface, sink, gate_stride, act)
    w = next(n for n in (64, 128, 256, 512, 1024) if rank <= n)
    return _op(iface, _launch("latent", f"kern_latent_rot_attn_{act}_w{w}", [128, 1, 1], [heads, "tokens" if ragged else "seqs", 1],
                              [*iface[:5], iface[6] if ragged else NULL[0], "i32", "i32", "i32", "i32", "f32", "out buffer<i32>", *iface[o:o + 3], *extra] + ["i32"] * 6,
                              [*map(P, range(5)), P(6) if ragged else NULL[1], I(heads), I(rank), I(table_width), I(page_size), {"f32": scale}, P(5),
                               *map(P, range(o, o + 3)), *more, I(rot_stride), I(rot), I(max_pos), I(int(halves)), I(window), I(gate_stride)],
                              shared_mem=(4 * rank + 8 + rot) * 4))


# ---- a residual with norms on both sides of a sublayer -----------------------------------------------------
def conv_line_bytes(width: int, taps: int, act: str = "bf16") -> int:
    """Bytes of the state line of a convolution over a row's inputs: its last taps - 1 rows."""
    return max(256, -(-(taps - 1) * width * ACT_BYTES[act] // 256) * 256)


def _conv_step(conv: tuple[int, int], act: str, at: int):
    """What a kernel that also convolves its row takes (`conv`: taps, bytes of a line): interface types, launch arguments."""
    types = ["in buffer<bf16>", f"out buffer<{act}>", "inout state", "in buffer<i32>"]
    return types, [(t, P(at + i)) for i, t in enumerate(types)] + [("i32", I(conv[0])), ("i64", L(conv[1]))]


def conv_add_op(width: int, taps: int, line_bytes: int, act: str = "bf16") -> dict:
    """Rows of a ragged call plus a causal convolution of them over time, channel by channel; the last taps - 1 rows of a sequence
    stay in its state line. Interface [h, w, out, state, lines, cu_seqlens, seqs, rows]."""
    iface = [f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{act}>", "inout state", "in buffer<i32>", "in buffer<i32>", "i32", "i32"]
    return _op(iface, _launch("conv_add", f"kern_conv_add_{act}", [256, 1, 1], [{"ceil_div": ["tokens", 4]}, -(-width // (1024 if width % 4 == 0 else 256)), 1],
                              [iface[0], *iface[2:6], iface[1], "i32", "i32", "i32", "i32", "i64"],
                              [P(0), *map(P, range(2, 6)), P(1), P(6), P(7), I(width), I(taps), L(line_bytes)]))


def resid_embed_op(width: int, vocab: int, eps: float, act: str = "bf16", scale: float = 1.0, conv: tuple[int, int] | None = None) -> dict:
    """Token row times `scale` into the f32 residual, and the first sublayer's normed input.
    Interface [ids, table, next norm w, x, xn, err]; `conv` (taps, bytes of a line; one row per sequence) also convolves the input:
    [conv w, convolved, state, lines] at the end."""
    iface = ["in buffer<i64>", "in buffer<bf16>", "in buffer<bf16>", "out buffer<f32>", f"out buffer<{act}>", "out buffer<i32>"]
    types, more = _conv_step(conv, act, 6) if conv else ([], [])
    return _op(iface + types, _launch("resid", f"kern_resid_embed_{'conv_' if conv else ''}{act}", [256, 1, 1], ["tokens", 1, 1],
                                      iface[:5] + ["i32", "i32", "f32", "f32", "out buffer<i32>"] + [t for t, _ in more],
                                      [*map(P, range(5)), I(width), I(vocab), {"f32": scale}, {"f32": eps}, P(5), *(a for _, a in more)], shared_mem=width * 4))


def resid_mix_op(width: int, eps: float, act: str = "bf16", routed: int = 0, last: bool = False) -> dict:
    """x += rms(y) w_post, and the next sublayer's normed input. Interface [x, y, w_post, w_next, xn], with `routed` (experts per
    token) also [perm, weights] at the end: y then holds expert-sorted rows. `last`: the sum goes to `hidden` and nothing is
    normed; interface [x, y, w_post, hidden]."""
    iface = ["in buffer<f32>" if last else "inout buffer<f32>", f"in buffer<{act}>", "in buffer<bf16>"]
    iface += ["out buffer<f32>"] if last else ["in buffer<bf16>", f"out buffer<{act}>"]
    n = len(iface)
    iface += ["in buffer<i32>", "in buffer<f32>"] if routed else []
    route = [(iface[n], P(n)), (iface[n + 1], P(n + 1))] if routed else [NULL, NULL]
    tail = [NULL, NULL, (iface[3], P(3))] if last else [(iface[3], P(3)), (iface[4], P(4)), NULL]
    parts = [(iface[0], P(0)), (iface[1], P(1)), *route, (iface[2], P(2)), *tail]
    return _op(iface, _launch("resid", f"kern_resid_mix_{act}", [256, 1, 1], ["tokens", 1, 1], [t for t, _ in parts] + ["i32", "i32", "f32"],
                              [a for _, a in parts] + [I(width), I(routed), {"f32": eps}], shared_mem=width * 4))


def resid_gate_op(width: int, eps: float, act: str = "bf16", routed: int = 0, last: bool = False, conv: tuple[int, int] | None = None) -> dict:
    """`resid_mix_op` of a result gated element by element: x += rms(y sigmoid(gate + b)) w_post. Interface [x, y, w_post, w_next, xn,
    gate, b] (`last`: [x, y, w_post, hidden, gate, b]), then with `routed` [perm, weights], with `conv` (taps, bytes of a line; one
    row per sequence) the next input convolved as well: [conv w, convolved, state, lines]."""
    iface = ["in buffer<f32>" if last else "inout buffer<f32>", f"in buffer<{act}>", "in buffer<bf16>"]
    iface += ["out buffer<f32>"] if last else ["in buffer<bf16>", f"out buffer<{act}>"]
    g = len(iface)
    iface += [f"in buffer<{act}>", "in buffer<bf16>"]
    n = len(iface)
    iface += ["in buffer<i32>", "in buffer<f32>"] if routed else []
    route = [(iface[n], P(n)), (iface[n + 1], P(n + 1))] if routed else [NULL, NULL]
    types, more = _conv_step(conv, act, len(iface)) if conv else ([], [])
    tail = [NULL, NULL, (iface[3], P(3))] if last else [(iface[3], P(3)), (iface[4], P(4))] + ([] if conv else [NULL])
    parts = [(iface[0], P(0)), (iface[1], P(1)), *route, (iface[2], P(2)), *tail, ("i32", I(width)), ("i32", I(routed)), ("f32", {"f32": eps}),
             (iface[g], P(g)), (iface[g + 1], P(g + 1)), *more]
    return _op(iface + types, _launch("resid", f"kern_resid_gate_{'conv_' if conv else ''}{act}", [256, 1, 1], ["tokens", 1, 1], [t for t, _ in parts],
                                      [a for _, a in parts], shared_mem=width * 4))


def resid_scale_op(width: int, eps: float, act: str = "bf16", *, routed: int = 0, bias: bool = False, shared_gate: int | None = None,
                   last: bool = False) -> dict:
    """x += s y element by element, and the next sublayer's normed input. Interface [x, y, s, w_next, xn] (`last`: [x, y, s, hidden],
    plus xn at the end of the list below when experts may hand back the input), then with `bias` [bias], with `routed` (experts
    per token) [perm, weights] — y holds expert-sorted rows, and a choice without a row stands for xn itself — and with
    `shared_gate` (the row stride of the gate's buffer) [shared rows, gate]: sigmoid(gate) weighs an expert of every token."""
    iface = ["in buffer<f32>" if last else "inout buffer<f32>", f"in buffer<{act}>", "in buffer<bf16>"]
    iface += ["out buffer<f32>"] if last else ["in buffer<bf16>", f"inout buffer<{act}>"]

    def more(*types):
        at = len(iface)
        iface.extend(types)
        return [(t, P(at + i)) for i, t in enumerate(types)]

    b = more("in buffer<bf16>") if bias else [NULL]
    route = more("in buffer<i32>", "in buffer<f32>") if routed else [NULL, NULL]
    sh = more(f"in buffer<{act}>", "in buffer<f32>") if shared_gate is not None else [NULL, NULL]
    if last:
        tail = [NULL, *(more(f"in buffer<{act}>") if routed else [NULL]), (iface[3], P(3))]
    else:
        tail = [(iface[3], P(3)), (iface[4], P(4)), NULL]
    parts = [(iface[0], P(0)), (iface[1], P(1)), *route, *sh, *b, (iface[2], P(2)), *tail]
    return _op(iface, _launch("resid", f"kern_resid_scale{'_routed' if routed else ''}_{act}", [256, 1, 1], ["tokens", 1, 1], [t for t, _ in parts] + ["i32", "i32", "i32", "f32"],
                              [a for _, a in parts] + [I(width), I(routed), I(shared_gate or 0), {"f32": eps}], shared_mem=width * 4))


# ---- linear attention with a decay per key channel -----------------------------------------------------------
LIN_CHUNK_MIN = 8       # rows of a call from which a sequence is computed in chunks
LIN_DIMS = 256          # most key channels of a head


def lin_line_bytes(heads: int, dk: int, dv: int, shifted: int = 0) -> tuple[int, int]:
    """(bytes of one per-sequence line, offset of S in it); `shifted`: columns of the kept previous row."""
    s_off = (shifted * 4 + 255) // 256 * 256
    return (s_off + heads * dk * dv * 4 + 255) // 256 * 256, s_off


def token_shift_op(width: int, targets: int, line_bytes: int, ragged: bool, act: str = "bf16") -> dict:
    """out[t, m] = h[t] + (h[t - 1] - h[t]) mu[m] for every target m; the row before a call's first is kept at the start of the
    state line (f32). Interface [h, mu, out, state, lines, (cu_seqlens,) seqs]."""
    iface = [f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{act}>", "inout state", "in buffer<i32>"] + (["in buffer<i32>"] if ragged else []) + ["i32"]
    cu_t, cu_a = (iface[5], P(5)) if ragged else NULL
    n = P(len(iface) - 1)
    cols = -(-width // 1024)
    shift = _launch("lin_attn", f"kern_token_shift_{act}", [256, 1, 1], ["tokens", cols, 1],
                    [*iface[:3], "in state" if ragged else "inout state", iface[4], cu_t, "i32", "i32", "i32", "i64"],
                    [*map(P, range(5)), cu_a, n, I(width), I(targets), L(line_bytes)])
    if not ragged:
        return _op(iface, shift)
    keep = _launch("lin_attn", f"kern_shift_state_{act}", [256, 1, 1], ["seqs", cols, 1], [iface[0], "inout state", iface[4], cu_t, "i32", "i32", "i64"],
                   [P(0), P(3), P(4), P(5), n, I(width), L(line_bytes)])
    return _op(iface, shift, keep)


def decay_op(n: int, rank: int, lda: int, kind: str, tau: float = 1.0, act: str = "f32") -> dict:
    """alpha [tokens, n] (f32) from a low-rank row a [tokens, rank]: `root` sigmoid(W a + b)^(1 / tau), `double_exp`
    exp(-exp(W tanh(a) + b)). Interface [a, w, bias, alpha, tokens]."""
    iface = [f"in buffer<{act}>", "in buffer<bf16>", "in buffer<bf16>", "out buffer<f32>", "i32"]
    return _op(iface, _launch("lin_attn", f"kern_decay_{act}", [256, 1, 1], [-(-n // 64), {"ceil_div": ["tokens", 64]}, 1], iface + ["i32"] * 4 + ["f32"],
                              [*map(P, range(5)), I(n), I(rank), I(lda), I({"root": 0, "double_exp": 1}[kind]), {"f32": 1.0 / tau}]))


def lin_fused(dv: int) -> bool:
    """Whether the step of a one-row call also norms and gates (a block then owns a head's whole row)."""
    return dv <= 128


def lin_rule_op(heads: int, dk: int, dv: int, stride: int, line_bytes: int, s_off: int, ragged: bool, act: str = "bf16", *, bonus: bool,
                q_scale: float = 1.0, fused: bool = False, norm_shared: bool = True, out_stride: int = 0, out_scale: float = 1.0,
                eps: float = 0.0, rows_max: int = 0, seqs_max: int = 0) -> dict:
    """S = diag(alpha) S + k v^T and its read by q. Interface [q, k, v, alpha, (u,) out, state, lines, (cu_seqlens,) seqs]; `fused`
    (out is then the normed, weighed and gated activation, else f32 rows) adds [gate, norm w] before the last. q, k, v and gate
    share their row stride. `rows_max`, `seqs_max`: the largest ragged call, which sizes what the chunks' preparation leaves behind."""
    if dk > LIN_DIMS:
        raise ValueError(f"{dk} key channels per head (at most {LIN_DIMS})")
    out_t = f"out buffer<{act if fused else 'f32'}>"
    parts = [("q", f"in buffer<{act}>"), ("k", f"in buffer<{act}>"), ("v", f"in buffer<{act}>"), ("alpha", "in buffer<f32>")]
    parts += [("u", "in buffer<bf16>")] if bonus else []
    parts += [("out", out_t), ("state", "inout state"), ("lines", "in buffer<i32>")]
    parts += [("cu", "in buffer<i32>")] if ragged else []
    parts += [("gate", f"in buffer<{act}>"), ("norm", "in buffer<bf16>")] if fused else []
    parts += [("seqs", "i32")]
    at = {n: (t, P(i)) for i, (n, t) in enumerate(parts)}
    pick = lambda *names: [at.get(n, NULL) for n in names]
    rk = next(r for r in (4, 8, 16, 32) if dk <= 8 * r)
    v = 1 if dv <= 32 else (2 if dv <= 64 else 4)
    chunked = ragged and act == "bf16" and not fused
    tb = 8 if ragged else 1
    args = pick("q", "k", "v", "gate", "alpha", "u", "norm", "out", "state", "lines", "cu", "seqs")
    rule = _launch("lin_attn", f"kern_lin_rule_{act}_r{rk}_v{v}", [256, 1, 1], [heads * -(-dv // (32 * v)), "seqs", 1],
                   [t for t, _ in args] + ["i32"] * 6 + ["i64"] + ["i32"] * 4 + ["f32"] * 3,
                   [a for _, a in args] + [I(heads), I(dk), I(dv), I(stride), I(0 if norm_shared else dv), I(out_stride), L(line_bytes), I(s_off), I(int(fused)),
                                           I(tb), I(LIN_CHUNK_MIN - 1 if chunked else C.I32_MAX), {"f32": q_scale}, {"f32": out_scale}, {"f32": eps}],
                   shared_mem=(3 * tb + 1) * dk * 4)
    iface = [t for _, t in parts]
    if not chunked:
        return _op(iface, rule)
    # a ragged call's long sequences in chunks on the tensor cores, its few-row ones (decode rows among prompts) row by row
    np_ = next(n for n in (32, 64, 128, 256) if dk <= n)
    block = 5 * 16 * (np_ + 8) * 2 + 3 * 16 * 24 * 2 + np_ * 4
    slots = rows_max // 16 + seqs_max + 1
    pick_t = lambda args: ([t for t, _ in args], [a for _, a in args])
    types, args = pick_t(pick("q", "k", "alpha", "u") + [("out buffer<u8>", {"scratch": "prep"})] + pick("cu", "seqs"))
    prep = _launch("lin_attn_chunk", f"kern_lin_prep_n{np_}", [128, 1, 1], [{"add": [{"ceil_div": ["tokens", 16]}, "seqs"]}, heads, 1], types + ["i32"] * 5 + ["f32"],
                   args + [I(heads), I(dk), I(stride), I(LIN_CHUNK_MIN), I(slots), {"f32": q_scale}], shared_mem=16 * np_ * 8 + np_ * 4)
    types, args = pick_t(pick("v") + [("in buffer<u8>", {"scratch": "prep"})] + pick("out", "state", "lines", "cu", "seqs"))
    chunk = _launch("lin_attn_chunk", f"kern_lin_chunk_n{np_}", [128, 1, 1], [heads * -(-dv // 64), "seqs", 1], types + ["i32"] * 4 + ["i64", "i32", "i32"],
                    args + [I(heads), I(dk), I(dv), I(stride), L(line_bytes), I(s_off), I(LIN_CHUNK_MIN)], shared_mem=4 * (block + 16 * 72 * 2))
    return _op(iface, prep, chunk, rule, scratch={"prep": {"dtype": "u8", "shape": [slots, heads * block]}})


def lin_norm_gate_op(heads: int, dv: int, gate_stride: int, norm_shared: bool, out_stride: int, out_scale: float, eps: float, act: str = "bf16") -> dict:
    """rms_norm per head of the f32 rows, times w (one per column, or shared by the heads), times silu(gate), times out_scale.
    Interface [o, gate, w, out]."""
    iface = ["in buffer<f32>", f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{act}>"]
    return _op(iface, _launch("lin_attn", f"kern_lin_norm_gate_{act}", [256, 1, 1], ["tokens", -(-heads // 8), 1], iface + ["i32"] * 5 + ["f32", "f32"],
                              [*map(P, range(4)), I(heads), I(dv), I(gate_stride), I(0 if norm_shared else dv), I(out_stride), {"f32": out_scale}, {"f32": eps}]))


# ---- attention in a sliding window ---------------------------------------------------------------------------
LOG2E = 1.4426950408889634


def qk_prep_op(hq: int, hk: int, d: int, dv: int, rot: int, page_size: int, row_stride: int, max_pos: int, eps: float, act: str = "bf16",
               halves: bool = False) -> dict:
    """Norm of q and k per head, rotary positions on the first `rot` columns (pairs of neighbours, or `halves`), k and v into the
    paged cache. Interface [qkv, state, positions, slots, cos, sin, q norm w, k norm w, err]."""
    if rot % 2 or rot > d:
        raise ValueError(f"rotary positions on {rot} of {d} columns")
    iface = [f"inout buffer<{act}>", "inout state", "in buffer<i64>", "in buffer<i64>", "in buffer<f32>", "in buffer<f32>", "in buffer<bf16>",
             "in buffer<bf16>", "out buffer<i32>"]
    return _op(iface, _launch("attn_window", f"kern_qk_prep_{act}", [256, 1, 1], ["tokens", 1, 1], iface[:8] + ["i32"] * 9 + ["f32", "out buffer<i32>"],
                              [*map(P, range(8)), I(hq), I(hk), I(d), I(dv), I(rot), I(int(halves)), I(page_size), I(row_stride), I(max_pos), {"f32": eps}, P(8)],
                              shared_mem=8 * max(d, dv) * 4))


def qk_prep_whole_op(hq: int, hk: int, d: int, dv: int, v_col: int, rot: int, page_size: int, row_stride: int, max_pos: int, eps: float, act: str = "bf16",
                     halves: bool = False) -> dict:
    """As `qk_prep_op` with norms over all columns of q and of k at once, and values from column `v_col` of the row, which may be
    the keys' own. Interface [qkv, state, positions, slots, cos, sin, q norm w, k norm w, err]."""
    if rot % 2 or rot > d:
        raise ValueError(f"rotary positions on {rot} of {d} columns")
    if (hq + hk) * d > 50000:
        raise ValueError(f"{hq} + {hk} heads of {d} columns (at most 50000 together)")
    iface = [f"inout buffer<{act}>", "inout state", "in buffer<i64>", "in buffer<i64>", "in buffer<f32>", "in buffer<f32>", "in buffer<bf16>",
             "in buffer<bf16>", "out buffer<i32>"]
    return _op(iface, _launch("attn_window", f"kern_qk_prep_whole_{act}", [256, 1, 1], ["tokens", 1, 1], iface[:8] + ["i32"] * 10 + ["f32", "out buffer<i32>"],
                              [*map(P, range(8)), I(hq), I(hk), I(d), I(dv), I(v_col), I(rot), I(int(halves)), I(page_size), I(row_stride), I(max_pos), {"f32": eps}, P(8)],
                              shared_mem=(hq + hk) * d * 4))


def window_tiles(hq: int, hk: int, d: int, dv: int, page_size: int, act: str) -> bool:
    """Whether windowed attention of this size runs on the tensor-core kernels."""
    return act == "bf16" and d == dv and d in (64, 128, 256) and hq // hk <= 16 and (page_size % 64 == 0 or (page_size % 8 == 0 and 64 % page_size == 0))


def _split_ranges(hk: int, seqs_max: int, reach: int | None) -> list[tuple[int, int, int]]:
    """(splits, fewest, most sequences) of a decode launch: enough sequences that heads x sequences x splits cover the SMs, and in a
    reach of so many keys at least two tiles a split."""
    ranges, hi, most = [], seqs_max, 8 if reach else 32
    for splits in (1, 2, 4, 8, 16, 32)[: 4 if reach else 6]:
        if reach and splits > 1 and splits * 128 > reach + 64:
            break
        lo = 1 if splits == most or (reach and 4 * splits * 64 > reach + 64) else max(1, -(-C.SMS // (hk * splits)))
        if lo <= hi:
            ranges.append((splits, lo, hi))
            hi = lo - 1
    if hi >= 1:
        s, lo, top = ranges.pop() if ranges else (1, 1, seqs_max)
        ranges.append((s, 1, top))
    return ranges


def _tiled_attn(form: str, iface: list, at: dict, maps: list, hq: int, hk: int, d: int, page_size: int, table_width: int, q_stride: int, out_stride: int, form_t: list,
                form_a: list, ragged: bool, seqs_max: int, reach: int | None, merge) -> dict:
    """The launches of one form (`window`, `sink`, `pooled`) of the paged attention bodies. `at`: where q, out, table and lens stand in
    the interface; `form_t` / `form_a`: what the form's entries take at their end; `merge(splits, ws_o, ws_ml)`: the launch that puts
    split keys together. Ragged calls add [cu_seqlens, work_p, count_p, work_d, count_d] to the interface."""
    g, q, out, table, lens = hq // hk, *(P(at[k]) for k in ("q", "out", "table", "lens"))
    q_t, out_t = iface[at["q"]], iface[at["out"]]
    map_t = ["bytes<128>"] * len(maps)
    lp = lambda ws, lists: map_t + [q_t, out_t] + (["out buffer<f32>"] * 2 if ws else ["i64"] * 2) + ["in buffer<i32>"] * 2 \
        + (["in buffer<i32>"] * 3 if lists else ["i64"] * 3) + ["i32"] * 8 + form_t
    sizes = lambda splits: [I(hq), I(hk), I(q_stride), I(out_stride), I(table_width), I(page_size), I(splits), I(C.I32_MAX)]
    if not ragged:
        ranges = _split_ranges(hk, seqs_max, reach)
        launches, most = [], max(s for s, _, _ in ranges)
        for splits, lo, hi in ranges:
            when = {"var": "seqs", **({"min": lo} if lo > 1 else {}), **({"max": hi} if hi < seqs_max else {})}
            kw = {"when": when} if len(when) > 1 else {}
            ws = [{"scratch": "ws_o"}, {"scratch": "ws_ml"}] if splits > 1 else [L(0), L(0)]
            launches.append(_launch("attn_window", f"kern_attn_{form}_decode_d{d}", [160, 1, 1], [hk, "seqs", splits], lp(splits > 1, False),
                                    [*maps, q, out, *ws, table, lens, L(0), L(0), L(0), *sizes(splits), *form_a], shared_mem=C.attn_smem(d), **kw))
            if splits > 1:
                launches.append(merge(splits, *ws) | kw)
        scratch = {"scratch": {"ws_o": {"dtype": "f32", "shape": ["seqs", hq * most * d]}, "ws_ml": {"dtype": "f32", "shape": ["seqs", hq * most * 2]}}} if most > 1 else {}
        return _op(iface, *launches, **scratch)
    o = len(iface)
    iface += ["in buffer<i32>"] * 5
    lists = [P(o + i) for i in range(5)]
    mode = C.attn_mode(hq, hk, d)
    few = {"var": "seqs", "max": C.FMHA_SEQS}
    many = {"var": "seqs", "min": C.FMHA_SEQS + 1}
    grid = lambda rows: [hk, {"add": [{"ceil_div": ["tokens", rows // g]}, "seqs"]}, 1]
    tail = [I(hq), I(hk), I(q_stride), I(out_stride), I(table_width), I(page_size), I(C.I32_MAX), *form_a]
    causal = lambda **kw: _launch("attn_fmha", f"kern_attn_{form}_fmha_d128", [192, 1, 1], grid(128), map_t + [q_t, out_t] + ["in buffer<i32>"] * 5 + ["i32"] * 7 + form_t,
                                  [*maps, q, out, table, lens, *lists[:3], *tail], shared_mem=768 + 128 * d * 2 + 128 * 64 * 2 + 2 * 2 * (64 * d * 2) + 256, **kw)
    listed = lambda kind, work, smem, g_, **kw: _launch("attn_window", f"kern_attn_{form}_{kind}_d{d}", [160, 1, 1], g_, lp(False, True),
                                                        [*maps, q, out, L(0), L(0), table, lens, lists[0], lists[work], lists[work + 1], *sizes(1), *form_a],
                                                        shared_mem=smem, **kw)
    one = lambda **kw: _launch("attn_window", f"kern_attn_{form}_ragged_d{d}", [160, 1, 1], grid(64), map_t + [q_t, out_t] + ["in buffer<i32>"] * 7 + ["i32"] * 7 + form_t,
                               [*maps, q, out, table, lens, *lists, *tail], shared_mem=C.attn_smem(d, prefill=True), **kw)
    rows = lambda **kw: listed("decode", 3, C.attn_smem(d), [hk, "seqs", 1], **kw)
    if mode == "auto":
        return _op(iface, causal(when=few), rows(when=few), one(when=many))
    if mode in ("fmha", "fmha2"):
        return _op(iface, causal(), rows())
    if mode == "ragged":
        return _op(iface, one())
    return _op(iface, listed("prefill", 1, C.attn_smem(d, prefill=True), grid(64)), rows())


def _head_width(d: int, dv: int) -> int:
    """The generic attention kernels' columns for heads of this size."""
    if max(d, dv) > 512:
        raise ValueError(f"heads of {d} / {dv} columns (at most 512)")
    return next(n for n in (64, 128, 256, 512) if max(d, dv) <= n)


def window_attn_op(hq: int, hk: int, d: int, dv: int, window: int, scale: float, cap: float, page_size: int, table_width: int, q_stride: int,
                   out_stride: int, out_scale: float, ragged: bool, act: str = "bf16", seqs_max: int = 0) -> dict:
    """Attention over the last `window` positions, capped scores, a sink per query head; rows times out_scale into columns of
    wider rows. Interface [q, state, out, block_table, lens, sink, err], then for ragged rows on the tensor cores (`window_tiles`)
    [cu_seqlens, work_p, count_p, work_d, count_d] as `attn_plan_op` fills them (lens per sequence), else [row_seq] (lens per row)."""
    if hq % hk:
        raise ValueError(f"{hq} query heads over {hk} key heads")
    iface = [f"in buffer<{act}>", "in state", f"out buffer<{act}>", "in buffer<i32>", "in buffer<i32>", "in buffer<bf16>", "out buffer<i32>"]
    if not window_tiles(hq, hk, d, dv, page_size, act):
        iface += ["in buffer<i32>"] if ragged else []
        row_t, row_a = (iface[7], P(7)) if ragged else NULL
        return _op(iface, _launch("attn_window", f"kern_window_attn_{act}_w{_head_width(d, dv)}", [128, 1, 1], [hq, "tokens" if ragged else "seqs", 1],
                                  [*iface[:5], row_t, iface[5], NULL[0]] + ["i32"] * 10 + ["f32"] * 3 + ["out buffer<i32>"],
                                  [*map(P, range(5)), row_a, P(5), NULL[1], I(hq), I(hk), I(d), I(dv), I(q_stride), I(out_stride), I(0), I(table_width), I(page_size),
                                   I(window), {"f32": scale}, {"f32": cap}, {"f32": out_scale}, P(6)], shared_mem=(4 * dv + 8) * 4))
    win_t = ["out buffer<i32>", "in buffer<bf16>", "i32", "f32", "f32", "f32"]
    win_a = [P(6), P(5), I(window), {"f32": 2 * LOG2E * scale / cap}, {"f32": cap * LOG2E}, {"f32": out_scale}]
    merge = lambda splits, ws_o, ws_ml: _launch(
        "attn_window", "kern_attn_window_merge", [min(256, d), 1, 1], [{"mul": ["seqs", hq]}, 1, 1],
        ["in buffer<f32>", "in buffer<f32>", iface[2], "in buffer<bf16>", NULL[0]] + ["i32"] * 6 + ["f32"],
        [ws_o, ws_ml, P(2), P(5), NULL[1], I(0), I(C.I32_MAX), I(hq), I(d), I(splits), I(out_stride), {"f32": out_scale}])
    return _tiled_attn("window", iface, {"q": 0, "out": 2, "table": 3, "lens": 4}, [C._kv_map(d, page_size, 1)], hq, hk, d, page_size, table_width, q_stride, out_stride,
                       win_t, win_a, ragged, seqs_max, window, merge)


# ---- attention with a sink and an output gate --------------------------------------------------------------------
def sink_attn_op(hq: int, hk: int, d: int, dv: int, scale: float, page_size: int, table_width: int, q_stride: int, out_stride: int, gate_stride: int,
                 ragged: bool, act: str = "bf16", *, sink: bool = False, seqs_max: int = 0) -> dict:
    """Causal attention whose softmax has one more score per query head in the denominator (`sink`: learned; else a score of 0),
    rows times sigmoid(gate). Interface [q, state, out, block_table, lens, gate, err, (sink)], then for ragged rows on the tensor
    cores (`window_tiles`) [cu_seqlens, work_p, count_p, work_d, count_d] as `attn_plan_op` fills them (lens per sequence), else
    [row_seq] (lens per row)."""
    if hq % hk:
        raise ValueError(f"{hq} query heads over {hk} key heads")
    iface = [f"in buffer<{act}>", "in state", f"out buffer<{act}>", "in buffer<i32>", "in buffer<i32>", f"in buffer<{act}>", "out buffer<i32>"]
    iface += ["in buffer<bf16>"] if sink else []
    sk, o = (("in buffer<bf16>", P(7)) if sink else NULL), len(iface)
    if not window_tiles(hq, hk, d, dv, page_size, act):
        iface += ["in buffer<i32>"] if ragged else []
        row_t, row_a = (iface[o], P(o)) if ragged else NULL
        return _op(iface, _launch("attn_window", f"kern_window_attn_{act}_w{_head_width(d, dv)}", [128, 1, 1], [hq, "tokens" if ragged else "seqs", 1],
                                  [*iface[:5], row_t, sk[0], iface[5]] + ["i32"] * 10 + ["f32"] * 3 + ["out buffer<i32>"],
                                  [*map(P, range(5)), row_a, sk[1], P(5), I(hq), I(hk), I(d), I(dv), I(q_stride), I(out_stride), I(gate_stride), I(table_width),
                                   I(page_size), I(C.I32_MAX), {"f32": scale}, {"f32": 0.0}, {"f32": 1.0}, P(6)], shared_mem=(4 * dv + 8) * 4))
    form_t, form_a = ["out buffer<i32>", sk[0], iface[5], "i32", "f32"], [P(6), sk[1], P(5), I(gate_stride), {"f32": scale * LOG2E}]
    merge = lambda splits, ws_o, ws_ml: _launch(
        "attn_window", "kern_attn_window_merge", [min(256, d), 1, 1], [{"mul": ["seqs", hq]}, 1, 1],
        ["in buffer<f32>", "in buffer<f32>", iface[2], sk[0], iface[5]] + ["i32"] * 6 + ["f32"],
        [ws_o, ws_ml, P(2), sk[1], P(5), I(gate_stride), I(C.I32_MAX), I(hq), I(d), I(splits), I(out_stride), {"f32": 1.0}])
    return _tiled_attn("sink", iface, {"q": 0, "out": 2, "table": 3, "lens": 4}, [C._kv_map(d, page_size, 1)], hq, hk, d, page_size, table_width, q_stride, out_stride,
                       form_t, form_a, ragged, seqs_max, None, merge)


# ---- attention in a window beside pooled blocks ------------------------------------------------------------------
def pooled_sizes(hk: int, d: int, dv: int, pool: int, page_size: int, act: str = "bf16") -> dict:
    """The second cache of attention with pooled blocks of `pool` tokens: a page of it holds the blocks that end in the page of the
    same number. -> slots of a page, bytes per token (what a state declares), bytes of a page."""
    slots = -(-page_size // pool)
    per = -(-slots * hk * (d + dv) * ACT_BYTES[act] // page_size)
    while per * page_size % 16:
        per += 1
    return {"slots": slots, "token": per, "page": per * page_size}


def pooled_tiles(hq: int, hk: int, d: int, dv: int, pool: int, page_size: int, act: str) -> bool:
    """Whether attention beside pooled blocks of this size runs on the tensor-core kernels: pages hold whole blocks or blocks whole
    pages, without gaps."""
    z = pooled_sizes(hk, d, dv, pool, page_size, act)
    slots = z["slots"]
    return window_tiles(hq, hk, d, dv, page_size, act) and (page_size % pool == 0 or pool % page_size == 0) and (slots % 64 == 0 or 64 % slots == 0) \
        and slots * hk * 2 * d * ACT_BYTES[act] == z["page"]


def qk_prep_pool_op(hq: int, hk: int, d: int, dv: int, rot: int, pool: int, page_size: int, table_width: int, row_stride: int, max_pos: int, ragged: bool,
                    act: str = "bf16", halves: bool = False) -> dict:
    """Rotary positions on the first `rot` columns of q and k, k and v into the paged cache, and the mean rows of the blocks that end
    here into the second. Interface [qkv, state, pooled state, positions, slots, block_table, cos, sin, err] (+ [cu_seqlens, seqs,
    rows] for ragged rows)."""
    if rot % 2 or rot > d:
        raise ValueError(f"rotary positions on {rot} of {d} columns")
    z = pooled_sizes(hk, d, dv, pool, page_size, act)
    iface = [f"inout buffer<{act}>", "inout state", "inout state", "in buffer<i64>", "in buffer<i64>", "in buffer<i32>", "in buffer<f32>", "in buffer<f32>",
             "out buffer<i32>"]
    smem = 8 * max(d, dv) * 4
    if not ragged:
        return _op(iface, _launch("attn_window", f"kern_qk_prep_pool_{act}", [256, 1, 1], ["tokens", 1, 1], iface[:8] + ["i32"] * 11 + ["i64", "i32", "out buffer<i32>"],
                                  [*map(P, range(8)), I(hq), I(hk), I(d), I(dv), I(rot), I(int(halves)), I(page_size), I(row_stride), I(max_pos), I(pool), I(z["slots"]),
                                   L(z["page"]), I(table_width), P(8)], shared_mem=smem))
    iface += ["in buffer<i32>", "i32", "i32"]
    prep = _launch("attn_window", f"kern_qk_prep_{act}", [256, 1, 1], ["tokens", 1, 1],
                   [*iface[:2], *iface[3:5], *iface[6:8], NULL[0], NULL[0]] + ["i32"] * 9 + ["f32", "out buffer<i32>"],
                   [P(0), P(1), P(3), P(4), P(6), P(7), NULL[1], NULL[1], I(hq), I(hk), I(d), I(dv), I(rot), I(int(halves)), I(page_size), I(row_stride), I(max_pos),
                    {"f32": 0.0}, P(8)], shared_mem=smem)
    means = _launch("attn_window", f"kern_pool_blocks_{act}", [256, 1, 1], ["tokens", 1, 1],
                    ["in state", "inout state", *iface[3:6], iface[9]] + ["i32"] * 8 + ["i64", "i32", "out buffer<i32>"],
                    [P(1), P(2), P(3), P(4), P(5), P(9), P(10), P(11), I(hk), I(d), I(dv), I(page_size), I(pool), I(z["slots"]), L(z["page"]), I(table_width), P(8)])
    return _op(iface, prep, means)


def pooled_attn_op(hq: int, hk: int, d: int, dv: int, window: int, pool: int, scale: float, page_size: int, table_width: int, q_stride: int, out_stride: int,
                   ragged: bool, act: str = "bf16", seqs_max: int = 0) -> dict:
    """Attention over the last `window` positions and the mean rows of all blocks of `pool` tokens that end before them, in one
    softmax. Interface [q, state, pooled state, out, block_table, lens, err], then for ragged rows on the tensor cores
    (`pooled_tiles`) [cu_seqlens, work_p, count_p, work_d, count_d] (lens per sequence), else [row_seq] (lens per row)."""
    if hq % hk:
        raise ValueError(f"{hq} query heads over {hk} key heads")
    z = pooled_sizes(hk, d, dv, pool, page_size, act)
    iface = [f"in buffer<{act}>", "in state", "in state", f"out buffer<{act}>", "in buffer<i32>", "in buffer<i32>", "out buffer<i32>"]
    if not pooled_tiles(hq, hk, d, dv, pool, page_size, act):
        iface += ["in buffer<i32>"] if ragged else []
        row_t, row_a = (iface[7], P(7)) if ragged else NULL
        return _op(iface, _launch("attn_window", f"kern_pooled_attn_{act}_w{_head_width(d, dv)}", [128, 1, 1], [hq, "tokens" if ragged else "seqs", 1],
                                  [*iface[:6], row_t] + ["i32"] * 11 + ["i64", "f32", "out buffer<i32>"],
                                  [*map(P, range(6)), row_a, I(hq), I(hk), I(d), I(dv), I(q_stride), I(out_stride), I(table_width), I(page_size), I(window), I(pool),
                                   I(z["slots"]), L(z["page"]), {"f32": scale}, P(6)], shared_mem=(4 * dv + 8) * 4))
    form_t, form_a = ["out buffer<i32>", "i32", "i32", "i32", "f32"], [P(6), I(window), I(pool), I(z["slots"]), {"f32": scale * LOG2E}]
    merge = lambda splits, ws_o, ws_ml: _launch(
        "attn_paged", "kern_attn_merge_splits", [min(256, d), 1, 1], [{"mul": ["seqs", hq]}, 1, 1], ["in buffer<f32>", "in buffer<f32>", iface[3]] + ["i32"] * 5,
        [ws_o, ws_ml, P(3), I(C.I32_MAX), I(hq), I(d), I(splits), I(out_stride)])
    return _tiled_attn("pooled", iface, {"q": 0, "out": 3, "table": 4, "lens": 5}, [C._kv_map(d, page_size, 1), C._kv_map(d, z["slots"], 2)], hq, hk, d, page_size,
                       table_width, q_stride, out_stride, form_t, form_a, ragged, seqs_max, window + table_width * page_size // pool, merge)


# ---- routed experts ---------------------------------------------------------------------------------------
def route_logits_op(experts: int, top: int, bias: bool = True) -> dict:
    """The `top` largest of logits + bias, weighed by the softmax over them. Interface [logits, (bias,) ids, weights, tokens]."""
    if not (1 <= top <= min(32, experts) and experts <= 1024):
        raise ValueError(f"{top} of {experts} experts per token (at most 32 of 1024)")
    iface = ["in buffer<f32>"] + (["in buffer<bf16>"] if bias else []) + ["out buffer<i32>", "out buffer<f32>", "i32"]
    b_t, b_a = (iface[1], P(1)) if bias else NULL
    o = 2 if bias else 1
    return _op(iface, _launch("moe", "kern_moe_route_logits", [128, 1, 1], [{"ceil_div": ["tokens", 4]}, 1, 1],
                              ["in buffer<f32>", b_t, "out buffer<i32>", "out buffer<f32>", "i32", "i32", "i32", "i32"],
                              [P(0), b_a, P(o), P(o + 1), P(o + 2), I(experts), I(top), I(experts)]))


def route_groups_op(experts: int, top: int, groups: int = 1, keep: int = 1, renorm: bool = False, *, softmax: bool = False,
                    correction: bool = False, group_top: int = 2, scale: float = 1.0, ld: int | None = None) -> dict:
    """Sigmoid scores, or their softmax; choices by the score plus a `correction` per expert: the `top` largest inside the best `keep`
    of equal groups of neighbours (a group's score: the sum of its `group_top` largest choices, two or one), weighing their
    scores, `renorm` divided by their sum, times `scale`. `ld`: row stride of the logits.
    Interface [logits, (correction,) ids, weights, tokens]."""
    if not (1 <= top <= min(32, keep * (experts // groups)) and experts <= 1024 and experts % groups == 0 and 1 <= keep <= groups <= 64):
        raise ValueError(f"{top} of {experts} experts per token in {keep} of {groups} groups (at most 32 of 1024, 64 groups)")
    iface = ["in buffer<f32>"] + (["in buffer<bf16>"] if correction else []) + ["out buffer<i32>", "out buffer<f32>", "i32"]
    b_t, b_a = (iface[1], P(1)) if correction else NULL
    o = 2 if correction else 1
    return _op(iface, _launch("moe", "kern_moe_route_groups", [128, 1, 1], [{"ceil_div": ["tokens", 4]}, 1, 1],
                              [iface[0], b_t, *iface[o:]] + ["i32"] * 7 + ["f32", "i32"],
                              [P(0), b_a, P(o), P(o + 1), P(o + 2), I(experts), I(top), I(groups), I(keep), I(int(softmax)), I(group_top), I(int(renorm)),
                               {"f32": scale}, I(ld or experts)], shared_mem=4 * (experts + groups) * 4))


def route_table_op(experts: int, top: int, vocab: int) -> dict:
    """No router: a table's row of the token id names its experts, each with weight 1 / top.
    Interface [token ids, table, ids, weights, tokens, err]."""
    if not 1 <= top <= min(32, experts):
        raise ValueError(f"{top} of {experts} experts per token (at most 32)")
    iface = ["in buffer<i64>", "in buffer<i32>", "out buffer<i32>", "out buffer<f32>", "i32", "out buffer<i32>"]
    return _op(iface, _launch("moe", "kern_moe_route_table", [256, 1, 1], [{"ceil_div": [{"mul": ["tokens", top]}, 256]}, 1, 1], iface[:5] + ["i32"] * 3 + [iface[5]],
                              [*map(P, range(5)), I(experts), I(top), I(vocab), P(5)]))


def routed_tile_rows(act: str, width: int, ff: int) -> int:
    """Rows of a tile of the planner's table: 128 for the tensor-core kernels, 64 for the generic one."""
    return C.BM if act == "bf16" and tiles_fit(width, ff) else 64


def routed_ops(width: int, ff: int, experts: int, top: int, tokens_max: int, act: str = "bf16", glu: str = "swiglu", limit: float = 0.0) -> dict:
    """plan / gather / fc1 / fc2 of routed experts with a gated unit (GLUS), under the interfaces of `moe._moe_ops`."""
    from . import moe

    cfg = moe.MoeConfig(hidden=width, moe_intermediate=ff, experts=experts, top_k=top, max_tokens=tokens_max)
    ops = moe._moe_ops(cfg, 0, experts, glu=glu, limit=limit)
    if routed_tile_rows(act, width, ff) == C.BM:
        return {k: ops[k] for k in ("moe_plan", "moe_gather", "moe_fc1", "moe_fc2")}
    bm = routed_tile_rows(act, width, ff)
    plan = ops["moe_plan"]["impl"]["launches"][0]
    plan["args"][9], plan["args"][10] = I(bm), I(tokens_max * top // bm + experts)
    b = f"buffer<{act}>"
    gather = _op(["in " + b, "in buffer<i32>", "out " + b, "i32"],
                 _launch("linear", f"kern_rows_scatter_{act}", [256, 1, 1], [{"mul": ["tokens", top]}, 1, 1],
                         ["in " + b, "in buffer<i32>", "out " + b, "i32", "i32", "i32"], [P(0), P(1), P(2), P(3), I(top), I(width)]))

    def routed(n, k, epi):
        return _op(["in " + b, "in buffer<bf16>", "out " + b, "in buffer<i32>", "in buffer<i32>", "i32", "out buffer<i32>"],
                   _launch("linear", f"kern_linear_grouped_{act}" + (f"_{epi}" if epi else ""), [256, 1, 1],
                           [-(-n // 64), {"clamp": [{"add": [{"ceil_div": [{"mul": ["tokens", top]}, bm]}, experts]}, 0, 4096]}, 1],
                           ["in " + b, "in buffer<bf16>", "out " + b, "in buffer<i32>", "in buffer<i32>", "i32", "i32", "i32", "i64", "out buffer<i32>", "f32"],
                           [P(0), P(1), P(2), P(3), P(4), P(5), I(n), I(k), L((2 if epi else 1) * n * k), P(6), {"f32": limit}]))

    return {"moe_plan": ops["moe_plan"], "moe_gather": gather, "moe_fc1": routed(ff, width, glu), "moe_fc2": routed(width, ff, "")}

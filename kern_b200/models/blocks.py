"""Op builders of the decoder blocks that take any size and either activation type (bf16, or f32 in a model's 32-bit
form): matrix products, hyper-connections, the Mamba-2 mixer, latent attention without positions, routed experts. Where a
bf16 size fits the tensor-core kernels the op is the one `common.py` builds; the rest runs the generic kernels of
linear.cu / ssd.cu / latent.cu. Weights are bf16 in both forms.
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


def tiles_fit(*extents: int) -> bool:
    """Whether rows of these lengths are whole 16-byte vectors of bf16, which the tensor-core tiles and TMA need."""
    return all(e % 8 == 0 for e in extents)


# ---- matrix products ----------------------------------------------------------------------------------
def _generic(sfx: str, iface, n: int, k: int, lda: int, ldc: int, rows_var: str, batch: int = 1, w=None, strides=(0, 0, 0)) -> dict:
    """`w`: (row stride, column stride) of the weights in elements; `strides`: what a step of the batch adds to A, W, C."""
    wsn, wsk = w or (k, 1)
    return _launch("linear", f"kern_linear_{sfx}", [256, 1, 1], [-(-n // 64), {"ceil_div": [rows_var, 64]}, batch],
                   iface[:3] + ["i32"] * 5 + ["i64"] * 5 + ["out buffer<i32>"],
                   [P(0), P(1), P(2), P(3), I(n), I(k), I(lda), I(ldc), L(wsn), L(wsk), *map(L, strides), P(4)])


def linear_op(n: int, k: int, *, act: str = "bf16", epilogue: str = "store", rows_var: str = "tokens", rows_max: int,
              lda: int | None = None, ldc: int | None = None) -> dict:
    """C[rows, n] = A[rows, k] . W[n, k]^T. Interface [a, w, c, rows, err]; epilogue store | f32 | swiglu as in `gemm_op`."""
    lda = k if lda is None else lda
    cols = n // 2 if epilogue == "swiglu" else n
    ldc = cols if ldc is None else ldc
    if act == "bf16" and tiles_fit(cols, k, lda, ldc):
        return C.gemm_op(n, k, epilogue=epilogue, rows_var=rows_var, rows_max=rows_max, lda=lda, ldc=ldc)
    out = "f32" if epilogue == "f32" else act
    sfx = act + {"store": "", "f32": "_f32" if act == "bf16" else "", "swiglu": "_swiglu"}[epilogue]
    iface = [f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{out}>", "i32", "out buffer<i32>"]
    return _op(iface, _generic(sfx, iface, cols, k, lda, ldc, rows_var))


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


def routed_tile_rows(act: str, width: int, ff: int) -> int:
    """Rows of a tile of the planner's table: 128 for the tensor-core kernels, 64 for the generic one."""
    return C.BM if act == "bf16" and tiles_fit(width, ff) else 64


def routed_ops(width: int, ff: int, experts: int, top: int, tokens_max: int, act: str = "bf16") -> dict:
    """plan / gather / fc1 / fc2 of routed SwiGLU experts under the interfaces of `moe._moe_ops`."""
    from . import moe

    cfg = moe.MoeConfig(hidden=width, moe_intermediate=ff, experts=experts, top_k=top, max_tokens=tokens_max)
    ops = moe._moe_ops(cfg, 0, experts)
    if routed_tile_rows(act, width, ff) == C.BM:
        return {k: ops[k] for k in ("moe_plan", "moe_gather", "moe_fc1", "moe_fc2")}
    bm = routed_tile_rows(act, width, ff)
    plan = ops["moe_plan"]["impl"]["launches"][0]
    plan["args"][9], plan["args"][10] = I(bm), I(tokens_max * top // bm + experts)
    b = f"buffer<{act}>"
    gather = _op(["in " + b, "in buffer<i32>", "out " + b, "i32"],
                 _launch("linear", f"kern_rows_scatter_{act}", [256, 1, 1], [{"mul": ["tokens", top]}, 1, 1],
                         ["in " + b, "in buffer<i32>", "out " + b, "i32", "i32", "i32"], [P(0), P(1), P(2), P(3), I(top), I(width)]))

    def routed(n, k, swiglu):
        return _op(["in " + b, "in buffer<bf16>", "out " + b, "in buffer<i32>", "in buffer<i32>", "i32", "out buffer<i32>"],
                   _launch("linear", f"kern_linear_grouped_{act}" + ("_swiglu" if swiglu else ""), [256, 1, 1],
                           [-(-n // 64), {"clamp": [{"add": [{"ceil_div": [{"mul": ["tokens", top]}, bm]}, experts]}, 0, 4096]}, 1],
                           ["in " + b, "in buffer<bf16>", "out " + b, "in buffer<i32>", "in buffer<i32>", "i32", "i32", "i32", "i64", "out buffer<i32>"],
                           [P(0), P(1), P(2), P(3), P(4), P(5), I(n), I(k), L((2 if swiglu else 1) * n * k), P(6)]))

    return {"moe_plan": ops["moe_plan"], "moe_gather": gather, "moe_fc1": routed(ff, width, True), "moe_fc2": routed(width, ff, False)}

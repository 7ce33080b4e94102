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


def head_linear_op(heads: int, n: int, k: int, *, act: str = "bf16", rows_max: int, lda: int, ldc: int, transposed: bool = False) -> dict:
    """Per head h: C[:, h n : (h + 1) n] = A[:, h k : (h + 1) k] . W_h^T, with W_h [n, k] stacked by head, or [k, n] when
    `transposed`. Interface [a, w, c, rows, err]."""
    iface = [f"in buffer<{act}>", "in buffer<bf16>", f"out buffer<{act}>", "i32", "out buffer<i32>"]
    return _op(iface, _generic(act, iface, n, k, lda, ldc, "tokens", heads, (1, n) if transposed else (k, 1), (k, n * k, n)))


def gate_mul_op(d: int, gate_stride: int, act: str = "bf16") -> dict:
    """out = x * sigmoid(gate). Interface [x, gate, out, tokens]."""
    iface = [f"in buffer<{act}>", f"in buffer<{act}>", f"out buffer<{act}>", "i32"]
    return _op(iface, _launch("linear", f"kern_gate_mul_{act}", [256, 1, 1], [{"ceil_div": [{"mul": ["tokens", d]}, 1024]}, 1, 1],
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

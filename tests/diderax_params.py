"""Parameter grids of the mechanism tests, shared by the CPU and the GPU file (kept to tuples of plain values)."""
from tests.barotar_params import ACTS, MANY

SIZES = (      # hq, hk, d, dv, page, sequences (context, new rows)
    (4, 2, 64, 64, 16, ((1, 1), (60, 60), (90, 3))),
    (16, 2, 128, 128, 16, ((150, 150), (33, 2), (70, 1))),
    (6, 2, 128, 128, 64, MANY),
    (16, 1, 64, 64, 64, MANY),
    (3, 3, 256, 256, 16, ((80, 70), (20, 1))),
    (2, 2, 128, 128, 64, ((200, 130), (64, 64))),
    (6, 2, 18, 18, 16, ((40, 33), (17, 1))),
    (3, 1, 40, 72, 16, ((50, 44), (3, 2))),
)
DECODE = (
    (4, 2, 64, 64, 16, ((1, 1), (64, 1), (65, 1), (90, 1))),
    (16, 2, 128, 128, 64, ((299, 1), (64, 1), (1, 1), (570, 1))),      # split keys, some with nothing in a split
    (8, 4, 128, 128, 16, tuple((1 + 31 * i % 200, 1) for i in range(41))),
    (3, 3, 256, 256, 16, ((80, 1), (20, 1))),
    (6, 2, 18, 18, 16, ((40, 1), (9, 1), (16, 1))),
)
LATENT = (      # heads, rank, rotated columns, page, sequences
    (5, 72, 16, 16, ((1, 1), (60, 41), (90, 3))),
    (17, 128, 64, 64, ((130, 70), (64, 64), (65, 1))),
    (2, 56, 8, 16, ((40, 33), (17, 1))),
    (16, 512, 64, 64, ((140, 20), (3, 3))),
    (4, 320, 40, 16, ((70, 10), (33, 2))),
    (3, 36, 6, 16, ((40, 33), (17, 1))),
    (2, 64, 96, 16, ((50, 12),)),
)
LATENT_DECODE = (
    (5, 72, 16, 16, ((1, 1), (60, 1), (90, 1))),
    (33, 128, 64, 64, ((130, 1), (64, 1), (65, 1), (600, 1))),
    (16, 512, 64, 64, tuple((1 + 31 * i % 200, 1) for i in range(40))),
    (2, 192, 64, 16, ((40, 1), (250, 1))),
    (4, 448, 64, 64, ((77, 1),)),
    (3, 36, 6, 16, ((40, 1), (17, 1))),
)
GRID = [
    ("rope_table", [(16, 1e4, 1.0), (64, 1e6, 8.0), (2, 10.0, 2.5)]),
    ("resid_scale", [(a, w, k) for a in ACTS for w in (64, 50, 1100) for k in ("plain", "bias", "routed", "identity", "shared")]),
    ("glu_bias", [(a, m, n, k) for a in ACTS for m, n, k in ((1, 64, 80), (4, 24, 40), (150, 72, 40), (300, 600, 64), (5, 33, 50))]),
    ("route", [(12, 3, 4, 2, 2.0), (16, 4, 4, 3, 0.5), (5, 2, 5, 3, 1.0), (8, 8, 2, 2, 1.5), (264, 8, 8, 4, 2.5), (6, 1, 1, 1, 1.0)]),
    ("routed_experts", [(a, *r) for a in ACTS for r in ((64, 32, 9, 3, 3, 3, 2, 150), (50, 11, 3, 3, 2, 2, 1, 70), (40, 144, 3, 1, 4, 2, 2, 1), (64, 24, 2, 6, 1, 1, 1, 40))]),
    ("prep", [(a, hq, hk, d, r, hv, t) for a in ACTS for hq, hk, d, r, hv, t in ((4, 2, 64, 32, True, True), (9, 3, 18, 18, True, True), (2, 1, 40, 2, True, False),
                                                                                (16, 2, 128, 128, True, True), (3, 1, 24, 8, False, True), (6, 2, 40, 12, True, True))]),
    ("attention", [(a, *s, True, False) for a in ACTS for s in SIZES] + [(a, *s, False, False) for a in ACTS for s in DECODE]
     + [("bf16", *SIZES[1], True, True), ("f32", *SIZES[6], True, True), ("bf16", *DECODE[1], False, True)]),
    ("latent_prep", [(a, *s) for a in ACTS for s in ((72, 16, 56), (36, 6, 22), (512, 64, 200))]),
    ("latent", [(a, *s, True) for a in ACTS for s in LATENT] + [(a, *s, False) for a in ACTS for s in LATENT_DECODE]),
]
ALL = [(name, args) for name, many in GRID for args in many]
IDS = [f"{n}-" + "-".join(str(x).replace(" ", "") for x in a if not isinstance(x, (list, tuple))) for n, a in ALL]

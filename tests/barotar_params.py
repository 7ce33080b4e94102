"""Parameter grids of the mechanism tests, shared by the CPU and the GPU file (kept to tuples of plain values)."""
ACTS = ("bf16", "f32")
CHUNKS3 = [(5, 1, 2, 9), (1, 4, 1, 1), (2, 2, 3, 20)]      # per sequence, per step
CHUNKS2 = [(5, 1, 70, 3, 16), (1, 2, 33, 66, 8)]
MANY = tuple((20 + 7 * i, r) for i, r in enumerate((1, 1, 5, 20, 1, 2, 33, 1, 1, 27)))      # more sequences than the few-sequence form takes
SIZES = (      # hq, hk, d, dv, window, page, sequences
    (4, 2, 64, 64, 21, 16, ((1, 1), (60, 60), (90, 3))),
    (16, 2, 128, 128, 50, 16, ((150, 150), (33, 2), (70, 1))),
    (6, 2, 128, 128, 70, 64, MANY),
    (16, 1, 64, 64, 9, 64, MANY),
    (3, 3, 256, 256, 33, 16, ((80, 70), (20, 1))),
    (2, 1, 128, 128, 1, 64, ((5, 5), (70, 66))),
    (2, 2, 128, 128, 500, 64, ((140, 130), (64, 64))),
    (6, 2, 18, 11, 9, 16, ((40, 33), (17, 1))),
    (3, 1, 40, 72, 20, 16, ((50, 44), (3, 2))),
)
DECODE = (
    (4, 2, 64, 64, 21, 16, ((1, 1), (21, 1), (22, 1), (90, 1))),
    (16, 2, 128, 128, 300, 64, ((299, 1), (300, 1), (301, 1), (570, 1))),      # split keys
    (8, 4, 128, 128, 65, 16, ((64, 1), (65, 1), (66, 1), (200, 1), (129, 1))),
    (3, 3, 256, 256, 33, 16, ((80, 1), (20, 1))),
    (6, 2, 18, 11, 9, 16, ((40, 1), (9, 1), (10, 1))),
)
GRID = [
    ("resid_embed", [(a, w) for a in ACTS for w in (64, 50, 300)]),
    ("resid", [(a, w, r) for a in ACTS for w, r in ((64, 0), (50, 0), (1100, 3), (33, 2), (40, 1))]),
    ("glu", [(a, m, n, k, e) for a in ACTS for m, n, k, e in ((3, 64, 80, "geglu"), (150, 72, 40, "geglu"), (300, 600, 64, "geglu"), (5, 33, 50, "geglu"), (9, 40, 24, "clamped"),
                                                          (70, 35, 21, "clamped"))]),
    ("route", [(40, 5, 4, 2), (12, 3, 3, 1), (10, 4, 10, 6), (9, 9, 1, 1), (256, 8, 8, 4)]),
    ("routed_experts", [(a, w, f, e, k, g, kp, n) for a in ACTS for w, f, e, k, g, kp, n in ((64, 32, 9, 3, 3, 2, 150), (50, 11, 6, 2, 2, 1, 70), (40, 144, 4, 1, 4, 2, 1))]),
    ("copy_cols", [()]),
    ("shift", [(a, w, t, CHUNKS3, True) for a in ACTS for w, t in ((64, 5), (37, 2), (1100, 3))] + [(a, w, t, [(1,) * 5] * 3, False) for a in ACTS for w, t in ((64, 5), (37, 1))]),
    ("decay", [(a, m, n, r, k) for a in ACTS for m, n, r, k in ((3, 70, 16, "root"), (130, 64, 5, "double_exp"), (1, 33, 64, "double_exp"), (65, 129, 33, "root"))]),
    ("rule", [(a, h, k, v, CHUNKS2, True, b) for a in ACTS for h, k, v in ((3, 24, 40), (2, 64, 64), (2, 7, 13)) for b in (False, True)]
     + [("bf16", h, k, v, CHUNKS2, True, b) for h, k, v in ((2, 128, 128), (1, 200, 24), (2, 32, 16)) for b in (False, True)]
     + [(a, h, k, v, [(1,) * 6] * 2, False, b) for a in ACTS for h, k, v in ((3, 24, 40), (2, 128, 128), (2, 7, 13), (1, 200, 150)) for b in (False, True)]),
    ("prep", [(a, hq, hk, d, dv, r, hv) for a in ACTS for hq, hk, d, dv, r, hv in ((4, 2, 64, 64, 32, False), (9, 3, 18, 11, 18, False), (2, 1, 40, 72, 2, False), (3, 1, 128, 128, 64, True))]),
    ("attention", [(a, *s, True) for a in ACTS for s in SIZES] + [(a, *s, False) for a in ACTS for s in DECODE]),
]
ALL = [(name, args) for name, many in GRID for args in many]
IDS = [f"{n}-" + "-".join(str(x).replace(" ", "") for x in a if not isinstance(x, (list, tuple))) for n, a in ALL]

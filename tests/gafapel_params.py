"""Parameter grids of the mechanism tests, shared by the CPU and the GPU file (kept to tuples of plain values)."""
ACTS = ("bf16", "f32")
CHUNKS3 = [(5, 1, 2, 9), (1, 4, 1, 1), (2, 2, 3, 20)]      # per sequence, per step
CHUNKS2 = [(5, 1, 70, 3), (1, 2, 33, 66)]
GRID = [
    ("embed", [(a, w, s) for a in ACTS for w, s in ((64, 4), (50, 1), (300, 7))]),
    ("hyper", [(a, w, s, r) for a in ACTS for w, s, r in ((64, 4, 0), (50, 1, 0), (72, 2, 3), (33, 3, 2), (40, 6, 1))]),
    ("row_norm", [(a,) for a in ACTS]),
    ("linear", [(a, m, n, k, e) for a in ACTS for m, n, k, e in ((3, 64, 80, "store"), (150, 72, 40, "store"), (5, 33, 50, "store"),
                                                                (9, 40, 24, "f32"), (70, 35, 21, "f32"), (130, 48, 56, "swiglu"), (2, 20, 30, "swiglu"))]),
    ("head_linear", [(a, m, h, n, k, t) for a in ACTS for m, h, n, k, t in ((3, 5, 72, 24, True), (140, 3, 40, 136, False), (17, 2, 33, 14, True),
                                                                          (1, 4, 64, 64, False), (200, 2, 128, 64, True))]),
    ("transpose", [()]),
    ("gate", [(a,) for a in ACTS]),
    ("route", [()]),
    ("routed_experts", [(a, w, f, e, k, n) for a in ACTS for w, f, e, k, n in ((64, 32, 9, 3, 150), (50, 11, 5, 2, 70), (40, 24, 4, 1, 1))]),
    ("conv_and_state", [(a, ch, t, CHUNKS3, True) for a in ACTS for ch, t in ((40, 4), (40, 2), (37, 3), (24, 6))]
     + [(a, ch, t, [(1,) * 7] * 3, False) for a in ACTS for ch, t in ((40, 4), (40, 3), (37, 2), (24, 6))]),
    ("ssd", [(a, h, p, n, g, CHUNKS2, True) for a in ACTS for h, p, n, g in ((4, 32, 48, 2), (3, 5, 7, 1), (2, 64, 130, 2))]
     + [("bf16", h, p, n, g, CHUNKS2, True) for h, p, n, g in ((4, 64, 128, 2), (2, 48, 64, 1), (3, 16, 16, 3))]
     + [(a, 4, 20, 24, 4, [(1,) * 5] * 2, False) for a in ACTS]),
    ("gate_norm", [(a, i, p) for a in ACTS for i, p in ((96, 4), (35, 7), (520, 1))]),
    ("append", [(a, r) for a in ACTS for r in (72, 36)]),
    ("attention", [(a, h, r, pg, lens, rag) for a in ACTS for h, r, pg, lens, rag in (
        (5, 72, 16, (1, 33, 160), True), (20, 200, 16, (17, 64), False), (3, 36, 16, (50, 16), True), (2, 512, 64, (130, 65), True),
        (17, 64, 64, (300, 1, 64), False))]),
]
ALL = [(name, args) for name, many in GRID for args in many]
IDS = [f"{n}-" + "-".join(str(x).replace(" ", "") for x in a if not isinstance(x, (list, tuple))) for n, a in ALL]

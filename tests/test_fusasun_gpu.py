"""The Fusasun decoder's kernels on a B200: every mechanism alone, and the whole model under every way of cutting its tokens
into calls, against the plain oracle (the same bodies as the CPU file, on longer sequences)."""
import pytest
import torch

from kern_b200.serve.scheduler import Request, Scheduler
from tests import fusasun_cases as A
from tests import fusasun_mechanisms as M
from tests import fusasun_params as P

pytestmark = pytest.mark.gpu


@pytest.mark.parametrize("name,args", P.ALL, ids=P.IDS)
def test_mechanism(cuda, name, args):
    getattr(M, name)(True, *args)


@pytest.mark.parametrize("mode", ("two", "ragged", "fmha2"))
def test_every_form_of_the_ragged_attention(cuda, monkeypatch, mode):
    """The forms that a call's size would not choose here, forced."""
    monkeypatch.setenv("KERN_B200_ATTN", mode)
    for size in (*P.SIZES[:4], *P.SIZES[5:7]):
        M.attention(True, "bf16", *size, True)


@pytest.mark.parametrize("dtype", P.ACTS)
@pytest.mark.parametrize("case", sorted(A.CASES))
def test_every_schedule_matches_the_oracle(cuda, case, dtype):
    cfg = A.config(case, dtype)
    w = A.weights(cfg)
    eng, truth = A.engine(cfg, w, True), A.Truth(cfg, w)
    prompts = A.prompts_of(cfg, (150, 1, 90, 33))
    for name, sched in A.schedules(prompts, cfg.page_size).items():
        rows = A.play(eng, truth, prompts, sched)
        assert A.within(rows, dtype), (name, float(rows.max()), float(rows.quantile(0.9)))
    assert eng.rt.check_guards() == []


@pytest.mark.parametrize("dtype", P.ACTS)
def test_long_decoding_over_page_window_and_block_borders(cuda, dtype):
    """400 positions, the last 80 decoded one by one; the same positions in portions. Pages of 64 as well."""
    for page in (16, 64):
        cfg = A.config("mixed", dtype, max_tokens=440, page_size=page)
        w = A.weights(cfg, seed=2)
        eng, truth = A.engine(cfg, w, True, tokens=640), A.Truth(cfg, w)
        prompts = A.prompts_of(cfg, (400,), seed=9)
        for sched in ([[("r0", 400)]], [[("r0", 320)]] + [[("r0", 1)]] * 80, [[("r0", n)] for n in A.portions(400, [63, 2, 64, 65, 7])]):
            rows = A.play(eng, truth, prompts, sched)
            assert A.within(rows, dtype), (page, float(rows.max()), float(rows.quantile(0.9)))


def test_scheduler_generates_what_the_oracle_would(cuda):
    cfg = A.config("mixed", "f32", max_tokens=24, max_seqs=3)
    w = A.weights(cfg)
    eng, truth = A.engine(cfg, w, True, slots=5), A.Truth(cfg, w)
    prompts = A.prompts_of(cfg, (30, 3, 19, 7, 26), seed=5)
    prompts["again"] = prompts["r0"] + [5, 6]
    sch = Scheduler(eng, max_seqs=3)
    reqs = [Request(id=r, prompt=p, max_tokens=6) for r, p in prompts.items()]
    for r in reqs:
        sch.submit(r)
    sch.run_until_idle(400)
    for r in reqs:
        ids = list(r.prompt)
        for _ in range(6):
            ids.append(int(truth.model.forward(ids, truth.model.new_cache())[-1].argmax()))
        assert r.out == ids[len(r.prompt):], r.id


def test_rows_alone_and_in_a_batch_agree(cuda):
    """bf16: the logits of a request's rows do not depend on what else is in the call, beyond rounding; twelve requests in one
    call take the many-sequence form of the attention, each alone the few-sequence one."""
    cfg = A.config("mixed", "bf16", max_tokens=400)
    w = A.weights(cfg)
    prompts = A.prompts_of(cfg, (60, 41, 7, 1, 25, 2, 30, 9, 1, 17, 66, 12), seed=4)
    eng = A.engine(cfg, w, True, tokens=100 * cfg.page_size, slots=14)
    alone = []
    for p in prompts.values():
        s = eng.open(len(p))
        alone.append(torch.as_tensor(eng.feed([(s, p)], [list(range(len(p)))])))
        eng.close(s)
    seqs = [eng.open(len(p)) for p in prompts.values()]
    both = torch.as_tensor(eng.feed(list(zip(seqs, prompts.values())), [list(range(len(p))) for p in prompts.values()]))
    rows = A.errors(both, torch.cat(alone).double())
    assert float(rows.quantile(0.9)) < 0.03 and float(rows.max()) < 0.1, (float(rows.max()), float(rows.quantile(0.9)))

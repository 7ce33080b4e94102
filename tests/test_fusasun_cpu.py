"""The Fusasun decoder on the host executor: every mechanism alone, and the whole model under every way of cutting its tokens
into calls, against the plain oracle."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from kern_b200.models import fusasun as G
from kern_b200.models import registry
from kern_b200.runtime import verify
from kern_b200.serve.scheduler import Request, Scheduler
from tests import fusasun_cases as A
from tests import fusasun_mechanisms as M
from tests import fusasun_params as P
from tests.oracles import fusasun as O

ROOT = Path(__file__).resolve().parent.parent


@pytest.mark.parametrize("name,args", P.ALL, ids=P.IDS)
def test_mechanism(name, args):
    getattr(M, name)(False, *args)


@pytest.mark.parametrize("dtype", P.ACTS)
@pytest.mark.parametrize("case", sorted(A.CASES))
def test_every_schedule_matches_the_oracle(case, dtype):
    cfg = A.config(case, dtype)
    w = A.weights(cfg)
    eng, truth = A.engine(cfg, w, False), A.Truth(cfg, w)
    prompts = A.prompts_of(cfg, (37, 1, 50, 18))
    for name, sched in A.schedules(prompts, cfg.page_size).items():
        rows = A.play(eng, truth, prompts, sched)
        assert A.within(rows, dtype), (name, float(rows.max()), float(rows.quantile(0.9)))


def test_wrong_readings_would_show(monkeypatch):
    """The oracle with one mechanism changed is far from the model: the limits above are sharp enough to see each."""
    cfg = A.config("mixed", "f32")
    w = A.weights(cfg)
    ids = A.prompts_of(cfg, (70,))["r0"]
    right = A.Truth(cfg, w)(ids)

    def layers(i, *path, value):
        out = json.loads(json.dumps(G.to_config(cfg)["layers"]))
        at = out[i]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        return out

    rot = ("mixer", "rot")
    for i, *path, value in ((0, *rot, "base", 9e3), (0, *rot, "dims", 30), (0, *rot, "scaling", "factor", 3.0), (0, *rot, "scaling", "low", 0.5), (0, *rot, "scaling", "high", 8.0),
                            (0, *rot, "scaling", "original", 80), (1, *rot, "base", 9e3), (1, *rot, "scaling", "factor", 2.5), (1, *rot, "scaling", "original", 400),
                            (1, *rot, "scaling", "fast", 1.2), (1, *rot, "scaling", "slow", 0.2), (2, "mixer", "scale", 0.12), (3, "mixer", "scale", 0.3),
                            (0, "mixer", "mask", "size", 21), (0, "mixer", "mask", "size", 19), (0, "mixer", "mask", "pool", 7), (2, "mixer", "mask", "size", 10),
                            (2, "mixer", "mask", "pool", 1 << 20), (1, "mixer", "mask", "size", 12), (1, "mixer", "mask", "size", 14), (3, "mixer", "mask", "size", 41)):
        t = A.Truth(cfg, w)
        t.model.c = {**t.model.c, "layers": layers(i, *path, value=value)}
        assert A.error(right, t(ids)) > 0.01, path
    for name in ("l0.canon1", "l2.canon1", "l0.rg1", "l1.rg2", "l2.rg1.b", "l0.rg2.b", "l1.mix.g", "l1.mix.dq.norm", "l3.mix.dkv.norm", "l0.mlp.table", "l3.mlp.table"):
        assert A.error(right, A.Truth(cfg, {**w, name: torch.zeros_like(w[name])})(ids)) > 0.01, name
    for where, change in (("embedding", {"scale": 1.0}), ("norm", {"eps": 1e-2})):
        t = A.Truth(cfg, w)
        t.model.c = {**t.model.c, where: change}
        assert A.error(right, t(ids)) > 0.005, where
    # tables without their factor, the gate after the norm, the gates and the residual gates fed with the convolved input
    yarn, gated, conv = O.yarn_frequencies, O.gated_sum, O.input_conv
    for name, other in (("yarn_frequencies", lambda *a: (yarn(*a)[0], 1.0)),
                        ("gated_sum", lambda x, y, h, w, b, post, eps: x + O.rms(y, eps) * post * O.sigmoid(h @ w.t() + b)),
                        ("input_conv", lambda w, h, st: conv(w, h, st) - h)):
        monkeypatch.setattr(O, name, other)
        assert A.error(right, A.Truth(cfg, w)(ids)) > 0.01, name
        monkeypatch.undo()


def test_registry_reads_a_folder_and_refuses_what_it_does_not_know(tmp_path):
    cfg = A.config("mixed")
    G.save_folder(tmp_path, cfg, A.weights(cfg))
    got, build = registry.from_folder(tmp_path, dtype="f32", max_seqs=3)
    assert got.dtype == "f32" and got.max_seqs == 3 and got.width == 72 and len(got.depth) == 4 and (got.taps, got.scale) == (4, 1.5)
    m, errs = verify(build(got))
    assert m is not None, errs[:3]
    doc = json.loads((tmp_path / "config.json").read_text())
    whole = json.loads(json.dumps(doc).replace("4.0", "4").replace("8.0", "8").replace("10000.0", "10000").replace("1.5", "1"))      # numbers without a point
    whole["layers"][0]["mixer"]["scale"] = whole["layers"][1]["mixer"]["scale"] = 1
    (tmp_path / "config.json").write_text(json.dumps(whole))
    for dtype in P.ACTS:
        m, errs = verify(build(registry.from_folder(tmp_path, dtype=dtype)[0]))
        assert m is not None, errs[:3]
    att, lat = doc["layers"][:2]
    but = lambda layer, **change: {"layers": [dict(layer, mixer={**layer["mixer"], **change})]}
    for change in ({"architecture": "Other"}, {"layers": [dict(att, type="attention2")]}, {"layers": [dict(att, mixer={"heads": 2})]}, {"layers": [dict(att, mlp={"kind": "dense"})]},
                   but(att, mask={"size": 4}), but(att, mask={"size": 4, "pool": 0}), but(att, mask={"size": 0, "pool": 2}), but(att, rot={"base": 1e4, "dims": 8, "scaling": {"factor": 2}}),
                   but(lat, rot_dim=8), but(lat, mask={}), {"layers": [dict(att, mlp={"kind": "moe", "router": {"experts": 4}})]}):
        (tmp_path / "config.json").write_text(json.dumps({**doc, **change}))
        with pytest.raises((KeyError, ValueError)):
            registry.from_folder(tmp_path)


@pytest.mark.parametrize("dtype", P.ACTS)
def test_manifests_of_the_built_in_shapes_verify(dtype):
    for cfg in (G.TINY_FUSASUN, G.FUSASUN_LARGE):
        m, errs = verify(registry.resolve(cfg.name, dtype=dtype)[1](registry.resolve(cfg.name, dtype=dtype)[0]))
        assert m is not None, errs[:3]


def greedy(truth, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(truth.model.forward(ids, truth.model.new_cache())[-1].argmax()))
    return ids[len(prompt):]


def test_scheduler_generates_what_the_oracle_would():
    """Greedy decoding of unequal requests through the scheduler: admissions, chunked prompts beside decode rows, slots and
    pages used again, a prefix that comes back from the cache."""
    cfg = A.config("mixed", "f32", max_tokens=24, max_seqs=3)
    w = A.weights(cfg)
    eng, truth = A.engine(cfg, w, False, slots=5), A.Truth(cfg, w)
    prompts = A.prompts_of(cfg, (30, 3, 19, 7, 26), seed=5)
    prompts["again"] = prompts["r0"] + [5, 6]
    sch = Scheduler(eng, max_seqs=3)
    reqs = [Request(id=r, prompt=p, max_tokens=6) for r, p in prompts.items()]
    for r in reqs:
        sch.submit(r)
    sch.run_until_idle(400)
    for r in reqs:
        assert r.out == greedy(truth, r.prompt, 6), r.id


def test_generate_and_sampling_fills():
    cfg = A.config("odd", "f32")
    w = A.weights(cfg)
    assert A.engine(cfg, w, False).generate([4, 9, 1], 5, chunk=2) == greedy(A.Truth(cfg, w), [4, 9, 1], 5)
    import dataclasses

    from kern_b200.engine import Sampling

    eng = A.engine(dataclasses.replace(cfg, sampling=True), w, False)
    assert eng.generate([4, 9, 1], 5) == greedy(A.Truth(cfg, w), [4, 9, 1], 5)               # temperature 0
    drawn = [eng.generate([4, 9, 1], 5, sampling=Sampling(temperature=200.0, seed=s)) for s in (1, 1, 2)]
    assert drawn[0] == drawn[1] and drawn[0] != drawn[2]


def test_replay_program_and_command_line(tmp_path):
    cfg = A.config("mixed")
    w = A.weights(cfg)
    G.save_folder(tmp_path / "m", cfg, w)
    truth = A.Truth(cfg, w)
    p = A.prompts_of(cfg, (70, 9))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p["r0"][:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p["r0"][66:67], "want": []}, {"id": "b", "tokens": p["r1"], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "b", "tokens": p["r1"][:8], "want": [7]}, {"id": "a", "tokens": p["r0"][67:], "want": [2, 0]}], "end": ["a", "b"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"),
                        "--max-tokens", "192", "--cpu"], input="\n".join(map(json.dumps, steps)), capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "o" / "1.f32").exists()
    got = [np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4").reshape(-1, cfg.vocab) for i in (0, 2)]
    a, b = truth(p["r0"]), truth(p["r1"])
    assert A.error(got[0], a[[0, 65]]) < A.LIMIT["f32"]
    assert A.error(got[1], torch.stack([b[7], a[69], a[67]])) < A.LIMIT["f32"]
    r = subprocess.run([sys.executable, "-m", "kern_b200", "run", "--model", str(tmp_path / "m"), "--dtype", "f32", "--cpu", "--prompt-ids", "4,9,1",
                        "--steps", "4"], capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.splitlines()[-1])["tokens"] == greedy(truth, [4, 9, 1], 4)


def test_pipeline_of_two_stages_emits_what_one_engine_does():
    """Cut at a layer boundary: the residual, the normed and the convolved input and the row plan cross; each state stays on its stage."""
    from kern_b200.cpu import CpuRuntime
    from kern_b200.serve import pp

    cfg = A.config("mixed", "f32")
    w = A.weights(cfg)
    doc = G.build_manifest(cfg)
    parts = pp.cut(doc, pp.layer_cuts(doc, 2))
    assert sorted(s for d in parts for s in d["states"]) == ["conv.l0", "conv.l1", "conv.l2", "conv.l3", "kv.l0", "kv.l1", "kv.l2", "kv.l3", "pool.l0", "pool.l2"]
    stages = [CpuRuntime(d, weights=w, tokens=cfg.page_size * 40, slots=4) for d in parts]
    for rt in stages:
        rt.once()
    single = A.engine(cfg, w, False)
    prompt, res = A.prompts_of(cfg, (22,))["r0"], []
    for eng in (single, pp.PipelineEngine(stages, single.p)):
        s = eng.open(40)
        eng.step([(s, prompt[:10])])
        out = [eng.step([(s, prompt[10:])])[0][0]]
        for _ in range(4):
            out.append(eng.step([(s, [out[-1]])])[0][0])
        res.append(out)
    assert res[0] == res[1]

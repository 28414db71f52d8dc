"""Rupasun on CPU in fp32: every mechanism and the whole serving path (step, cache, engine, scheduler,
command line, trace runner) against the plain implementation."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_rupasun as plain
import rupasun_cases as cases
from coeus_b200.foundation.error import Error
from coeus_b200.models import hybrid as H
from coeus_b200.models import registry
from coeus_b200.ops import ragged as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_benches = {}


def bench(kind):
    if kind not in _benches:
        _benches[kind] = cases.Bench(kind, "cpu", torch.float32)
    return _benches[kind]


@pytest.mark.parametrize("check", cases.MECHANISM_CHECKS, ids=lambda c: c.__name__[6:])
def test_mechanism(check):
    check("cpu", torch.float32, 2e-5)


@pytest.mark.parametrize("kind", ["odd", "wide", "large"])
@pytest.mark.parametrize("check", cases.MODEL_CHECKS, ids=lambda c: c.__name__[6:])
def test_model(kind, check):
    check(bench(kind))


def test_plain_window_counts_the_position_itself():
    seen = [[j for j in range(8) if plain.visible(i, j, 3)] for i in range(5)]
    assert seen == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4]]


def test_plain_rotations_keep_distances():
    x = cases.rnd((9, 2, 6), 1, "cpu").double()
    for turn in (plain.rotate_halves, plain.rotate_pairs):
        y = turn(x, 4, 7.0)
        assert torch.equal(y[..., 4:], x[..., 4:]) and torch.equal(y[0], x[0])
        assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1))
        z = turn(x[:1].expand(9, 2, 6).contiguous(), 4, 7.0)          # scores depend on the distance only
        assert torch.allclose((z[5] * z[2]).sum(-1), (z[8] * z[5]).sum(-1))
    e = torch.zeros(2, 1, 4, dtype=torch.float64)
    e[:, :, 0] = 1
    assert torch.allclose(plain.rotate_halves(e, 4, 7.0)[1, 0], torch.tensor([math.cos(1), 0, math.sin(1), 0]).double())
    assert torch.allclose(plain.rotate_pairs(e, 4, 7.0)[1, 0], torch.tensor([math.cos(1), math.sin(1), 0, 0]).double())


def test_plain_choice_respects_groups():
    z = torch.tensor([9.0, -9, -9, 1, 1, 1.1, -9, 8, -9], dtype=torch.float64)     # groups: 1 big, 3 fair, 1 big
    chosen, weight = plain.choose(z, 2, 3, 1, 2.0)
    assert set(chosen) == {5, 3} or set(chosen) == {5, 4}
    assert abs(float(weight.sum()) - 2.0) < 1e-12
    assert plain.choose(z, 2, 1, 1, 1.0)[0] == [0, 7]
    assert plain.choose(z, 3, 3, 2, 1.0)[0][0] == 0


@pytest.mark.parametrize("kind", ["odd", "wide", "large"])
def test_directory_round_trip_and_registry(kind, tmp_path):
    b = bench(kind)
    registry.save_dir(b.lm, str(tmp_path))
    config = registry.read_config(str(tmp_path))
    assert {e["type"] for e in config["layers"]} == {"attention", "attention_2"}
    assert registry.resolve(config).name == "Rupasun" and "Rupasun" in registry.architectures()
    lm = registry.load_dir(str(tmp_path), device="cpu", dtype=torch.float32)
    assert lm.cfg == b.cfg and lm.num_parameters() == b.lm.num_parameters()
    got = lm.state_dict()
    assert set(got) == set(b.w)
    for n in b.w:
        assert got[n].shape == b.w[n].shape and torch.equal(got[n].float(), b.w[n].float()), n
    with pytest.raises(Error):
        registry.load_dir(str(tmp_path), device="cpu", training=True)
    with pytest.raises(Error):
        H.load_hybrid({k: v for k, v in b.w.items() if k != "l0.mix.lq2"}, config, device="cpu")
    with pytest.raises(Error):
        H.load_hybrid({**b.w, "l1.mix.g": torch.zeros(5)}, config, device="cpu")


def test_config_is_checked():
    j = H.config_to_json(cases.config("odd"))
    assert H.config_from_json(j, {}) == cases.config("odd")

    def broken(edit):
        c = json.loads(json.dumps(j))
        edit(c)
        with pytest.raises(Error):
            H.config_from_json(c, {})
    mixer = lambda n, **kw: lambda c: c["layers"][n]["mixer"].update(kw)        # noqa: E731
    broken(lambda c: c["layers"][0].update(type="mamba2"))
    broken(lambda c: c.update(architecture="Bananex"))              # a design without these mixers
    broken(lambda c: c.update(architecture="Other"))
    broken(mixer(0, kv_heads=4))
    broken(mixer(0, dim=300))
    broken(mixer(0, rot=dict(dims=5, base=10.0)))
    broken(mixer(0, rot=dict(dims=12, base=10.0)))
    broken(mixer(1, mask=dict(size=0)))
    broken(mixer(1, softcap=0.0))
    mlp = lambda n, part, **kw: lambda c: c["layers"][n]["mlp"][part].update(kw)   # noqa: E731
    broken(lambda c: c["layers"][1]["mlp"].update(kind="sparse"))
    broken(lambda c: c["layers"][1]["mlp"].update(ff=0))
    broken(mlp(0, "router", top=5))
    broken(mlp(0, "router", experts=7))
    broken(mlp(0, "router", groups=dict(count=3, keep=4)))
    broken(mlp(0, "expert", limit=0.0))
    broken(mlp(0, "shared", ff=0))


def _run(args, **kw):
    return subprocess.run([sys.executable, *args], capture_output=True, text=True, timeout=300,
                          cwd=ROOT, **kw)


def test_command_line(tmp_path):
    b = bench("odd")
    registry.save_dir(b.lm, str(tmp_path))
    prompt = cases.tokens(b.cfg, 9, 4)
    r = _run(["-m", "coeus_b200", "generate", "--device=cpu", f"--weights={tmp_path}",
              "--prompt_ids=" + ",".join(map(str, prompt)), "--max_tokens=6"])
    assert r.returncode == 0, r.stderr
    out = json.loads(r.stdout.strip().splitlines()[-1])
    cases.agrees(b, prompt, out["token_ids"])
    r = _run(["-m", "coeus_b200", "info", f"--weights={tmp_path}"])
    assert json.loads(r.stdout.strip().splitlines()[-1])["architecture"] == "Rupasun"


def test_trace_runner(tmp_path):
    """Steps on standard input, logits in files; slots and pages used again, one request left out for
    a step, portions down to two tokens."""
    b = bench("odd")
    registry.save_dir(b.lm, str(tmp_path / "m"))
    out = tmp_path / "out"
    out.mkdir()
    seqs = {"a": cases.tokens(b.cfg, 33, 33), "b": cases.tokens(b.cfg, 70, 8)}
    plan = [([("a", 20, [0, 19])], []), ([("b", 64, []), ("a", 1, [0])], []),
            ([("b", 2, [1, 0])], []), ([("a", 12, [11]), ("b", 4, [3])], ["a", "b"]),
            ([("b#2", 70, [69, 5])], ["b#2"])]
    at, lines, want = {}, [], {}
    for n, (entries, end) in enumerate(plan):
        es, rows = [], []
        for i, m, w in entries:
            lo = at.get(i, 0)
            ids = seqs[i.split("#")[0]]
            es.append({"id": i, "tokens": ids[lo:lo + m], "want": w})
            rows += [b.oracle(ids)[lo + k] for k in w]
            at[i] = lo + m
        lines.append(json.dumps({"step": n, "entries": es, "end": end}))
        if rows:
            want[n] = torch.stack(rows)
    r = _run(["bin/trace_run", "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(out),
              "--max-tokens", "192", "--device", "cpu"], input="\n".join(lines) + "\n")
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:5] == [f"done {n}" for n in range(5)]
    for n, rows in want.items():
        got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(rows), -1)
        b.close(torch.from_numpy(got), rows)


def test_batches_cut_windows_without_pieces_into_tiles():
    """Long entries whose heads the piece kernel does not take, under a window and without one."""
    for plan, tiles in ((R.AttnPlan(None, False, 9), 4), (R.AttnPlan(None, False), 4),
                        (R.AttnPlan(None, False, 9, tiles=False), 0)):
        b = R.RaggedBatch([R.Entry(0, 30, [0] * 200), R.Entry(1, 5, [0])], "cpu", plans=[plan])
        assert b.plans[plan][0] == tiles and b.plans[plan][1] == 0

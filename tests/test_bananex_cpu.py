"""Bananex on CPU in fp32: every mechanism and the whole serving path (step, cache, state, engine,
scheduler, command line, trace runner) against the plain implementation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import bananex_cases as cases
import plain_bananex as plain
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


@pytest.mark.parametrize("kind", ["odd", "state", "latent"])
@pytest.mark.parametrize("check", cases.MODEL_CHECKS, ids=lambda c: c.__name__[6:])
def test_model(kind, check):
    check(bench(kind))


def test_plain_window_counts_the_position_itself():
    seen = [[j for j in range(8) if plain.window_visible(i, j, 3)] for i in range(5)]
    assert seen == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4]]


def test_plain_orders_the_loop():
    cfg = {"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}
    assert plain.order(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert plain.order({"layers": [0] * 2}) == [(0, None), (1, None)]
    odd = cases.config("odd")
    assert [tuple(r) for r in odd.runs()] == plain.order(H.config_to_json(odd))


@pytest.mark.parametrize("kind", ["odd", "wide", "state"])
def test_directory_round_trip_and_registry(kind, tmp_path):
    b = bench(kind)
    registry.save_dir(b.lm, str(tmp_path))
    config = registry.read_config(str(tmp_path))
    assert registry.resolve(config).name == "Bananex" and "Bananex" in registry.architectures()
    lm = registry.load_dir(str(tmp_path), device="cpu", dtype=torch.float32)
    assert lm.cfg == b.cfg and lm.num_parameters() == b.lm.num_parameters()
    got = lm.state_dict()
    assert set(got) == set(b.w)
    for n in b.w:
        assert got[n].shape == b.w[n].shape and torch.equal(got[n].float(), b.w[n].float()), n
    with pytest.raises(Error):
        registry.load_dir(str(tmp_path), device="cpu", training=True)
    with pytest.raises(Error):
        H.load_hybrid({k: v for k, v in b.w.items() if k != "l1.norm1b"}, config, device="cpu")
    with pytest.raises(Error):
        H.load_hybrid({**b.w, "l0.shift": torch.zeros(5)}, config, device="cpu")


def test_config_is_checked():
    j = H.config_to_json(cases.config("odd"))
    assert H.config_from_json(j, {}) == cases.config("odd")

    def broken(edit):
        c = json.loads(json.dumps(j))
        edit(c)
        with pytest.raises(Error):
            H.config_from_json(c, {})
    broken(lambda c: c["layers"][0].update(type="other"))
    broken(lambda c: c.update(architecture="Sapasun"))              # a design without these mixers
    broken(lambda c: c["layers"][0]["mixer"].update(groups=4))
    broken(lambda c: c["layers"][0]["mixer"].update(norm_groups=4))
    broken(lambda c: c["layers"][0]["mixer"].update(conv=40))
    broken(lambda c: c["layers"][1]["mixer"].update(rot_dim=5))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4))
    broken(lambda c: c["layers"][1]["mixer"]["mask"].update(size=0))
    broken(lambda c: c["layers"][1]["mixer"].update(kv_rank=4000))
    broken(lambda c: c["layers"][2]["mixer"].update(width=0))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda c: c["loop"].update(stop=9))
    broken(lambda c: c["loop"].update(times=0))


def _run(args, **kw):
    return subprocess.run([sys.executable, *args], capture_output=True, text=True, timeout=300,
                          cwd=ROOT, **kw)


def test_command_line(tmp_path):
    b = bench("state")
    registry.save_dir(b.lm, str(tmp_path))
    prompt = cases.tokens(b.cfg, 9, 4)
    r = _run(["-m", "coeus_b200", "generate", "--device=cpu", f"--weights={tmp_path}",
              "--prompt_ids=" + ",".join(map(str, prompt)), "--max_tokens=6"])
    assert r.returncode == 0, r.stderr
    out = json.loads(r.stdout.strip().splitlines()[-1])
    cases.agrees(b, prompt, out["token_ids"])
    r = _run(["-m", "coeus_b200", "info", f"--weights={tmp_path}"])
    assert json.loads(r.stdout.strip().splitlines()[-1])["architecture"] == "Bananex"


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

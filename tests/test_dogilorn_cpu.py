"""Dogilorn on CPU in fp32: every mechanism and the whole serving path (step, cache, state, engine, scheduler,
command line, trace runner) against the plain implementation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import dogilorn_cases as cases
import plain_dogilorn as plain
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


def test_plain_window_keeps_the_first_positions():
    seen = [[j for j in range(9) if plain.visible(i, j, 3, 2)] for i in range(8)]
    assert seen[:4] == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3]]
    assert seen[4:] == [[0, 1, 2, 3, 4], [0, 1, 3, 4, 5], [0, 1, 4, 5, 6], [0, 1, 5, 6, 7]]
    assert [j for j in range(9) if plain.visible(1, j, 3, 5)] == [0, 1]
    assert [j for j in range(9) if plain.visible(7, j, 3)] == [5, 6, 7]


def test_plain_softmax_beside_one():
    s = torch.tensor([[0.0, 0.0], [3.0, -float("inf")]], dtype=torch.float64)
    p = plain.weights_beside_one(s)
    assert torch.allclose(p[0], torch.full((2,), 1 / 3, dtype=torch.float64))
    e = float(torch.tensor(3.0).double().exp())
    assert abs(float(p[1, 0]) - e / (1 + e)) < 1e-12 and float(p[1, 1]) == 0


def test_plain_convolution_and_norm():
    h = torch.arange(8, dtype=torch.float64).view(4, 2)
    taps = torch.tensor([[1.0, 10.0], [0.0, 0.5]], dtype=torch.float64)
    assert plain.conv_in(h, taps).tolist() == [[0, 1.5], [22, 4.5], [46, 7.5], [70, 10.5]]
    y = plain.layer_norm(h, torch.ones(2), torch.tensor([0.0, 1.0]), 0.0)
    assert torch.allclose(y, torch.tensor([-1.0, 2.0]).double().expand(4, 2))


def test_plain_choice():
    s = torch.tensor([0.1, 0.2, 0.05, 0.3, 0.25, 0.1], dtype=torch.float64)
    z = s.log()
    zero = torch.zeros(6, dtype=torch.float64)
    assert plain.choose(z, zero, 2, 1, 1)[0] == [3, 4]
    chosen, weight = plain.choose(z, zero - 0.5, 3, 2, 1)          # every choice score is negative
    assert chosen == [3, 4, 5] and torch.allclose(weight, s[3:])
    lift = zero.clone()
    lift[2] = 1.0
    assert plain.choose(z, lift, 2, 3, 2)[0] == [2, 3] and plain.choose(z, lift, 2, 2, 1)[0] == [2, 1]


@pytest.mark.parametrize("kind", ["odd", "wide", "large"])
def test_directory_round_trip_and_registry(kind, tmp_path):
    b = bench(kind)
    registry.save_dir(b.lm, str(tmp_path))
    config = registry.read_config(str(tmp_path))
    assert {e["type"] for e in config["layers"]} == {"attention"}
    assert {e["mlp"]["kind"] for e in config["layers"] if e["mlp"]} == {"dense", "moe"}
    assert registry.resolve(config).name == "Dogilorn" and "Dogilorn" in registry.architectures()
    lm = registry.load_dir(str(tmp_path), device="cpu", dtype=torch.float32)
    assert lm.cfg == b.cfg and lm.num_parameters() == b.lm.num_parameters()
    got = lm.state_dict()
    assert set(got) == set(b.w) and "head" not in got
    for n in b.w:
        assert got[n].shape == b.w[n].shape and torch.equal(got[n].float(), b.w[n].float()), n
    with pytest.raises(Error):
        registry.load_dir(str(tmp_path), device="cpu", training=True)
    with pytest.raises(Error):
        H.load_hybrid({k: v for k, v in b.w.items() if k != "l0.mix.k.norm"}, config, device="cpu")
    with pytest.raises(Error):
        H.load_hybrid({**b.w, "l1.canon1": torch.zeros(5)}, config, device="cpu")


def test_layers_that_share_keys_have_no_tensors_for_them():
    names = H.tensor_shapes(cases.config("odd"))
    assert {n[7:] for n in names if n.startswith("l2.mix.")} == {"q", "q.norm", "temp", "o"}
    assert {n[7:] for n in names if n.startswith("l0.mix.")} == {"q", "k", "v", "q.norm", "k.norm", "temp", "o"}


def test_optional_parts_of_a_configuration():
    """No groups, no identity experts, no shared expert, no mask, no rotation, no kept positions."""
    j = H.config_to_json(cases.config("odd"))
    for key in ("groups", "identity"):
        j["layers"][3]["mlp"]["router"].pop(key, None)
    cfg = H.config_from_json(j, {})
    m = cfg.layers[3].mlp
    assert (m.groups, m.keep, m.identity, m.shared) == (1, 1, 0, None)
    assert H.config_to_json(cfg) == H.config_to_json(cases.config("odd"))
    a = H.config_to_json(cases.config("large"))["layers"][0]["mixer"]
    assert "mask" not in a and "rot" not in j["layers"][3]["mixer"] and "kv_from" not in a


def test_config_is_checked():
    j = H.config_to_json(cases.config("odd"))
    assert H.config_to_json(H.config_from_json(j, {})) == j

    def broken(edit):
        c = json.loads(json.dumps(j))
        edit(c)
        with pytest.raises(Error):
            H.config_from_json(c, {})
    mixer = lambda n, **kw: lambda c: c["layers"][n]["mixer"].update(kw)        # noqa: E731
    broken(lambda c: c["layers"][0].update(type="mamba2"))
    broken(lambda c: c["canon"].update(taps=0))
    broken(lambda c: c["canon"].update(taps=40))
    broken(mixer(0, kv_heads=4))
    broken(mixer(0, dim=300))
    broken(mixer(0, rot=dict(dims=5, base=10.0)))
    broken(mixer(1, mask=dict(size=0)))
    broken(mixer(1, mask=dict(size=4, keep_first=-1)))
    broken(mixer(2, kv_from=2))                                     # itself
    broken(mixer(2, kv_from=3))                                     # a later layer
    broken(mixer(2, kv_from=1))                                     # other heads
    broken(mixer(4, kv_from=2))                                     # a layer without keys of its own
    mlp = lambda n, part, **kw: lambda c: c["layers"][n]["mlp"][part].update(kw)   # noqa: E731
    broken(lambda c: c["layers"][1]["mlp"].update(kind="sparse"))
    broken(lambda c: c["layers"][1]["mlp"].update(ff=0))
    broken(lambda c: c["layers"][1]["mlp"].update(limit=0.0))
    broken(mlp(0, "router", top=7))
    broken(mlp(0, "router", experts=7))
    broken(mlp(0, "router", identity=4))
    broken(mlp(0, "router", identity=300))
    broken(mlp(0, "router", groups=dict(count=3, keep=4)))
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
    assert json.loads(r.stdout.strip().splitlines()[-1])["architecture"] == "Dogilorn"


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


def test_batches_name_the_kept_keys_of_a_piece():
    """Pieces of a window: where the first positions' keys lie, and whether a row's window has passed them."""
    plan = R.AttnPlan(None, True, 100, keep=5)

    def pieces(*entries):
        b = R.RaggedBatch([R.Entry(s, p, [0] * n) for s, p, n in entries], "cpu", plans=[plan])
        _, n, _, extra, rec, where = b.plan(plan)[:6]
        return rec.view(n, 8).tolist(), where.view(extra, 2).tolist()
    rec, where = pieces((0, 0, 300), (1, 0, 90))
    assert sorted(rec) == [[0, 256, 0, 0, 0, 5, 0, 0], [256, 44, 157, 99, 0, 5, 157, 0], [300, 90, 300, 0, 300, 0, 0, 0]]
    assert where == []
    rec, where = pieces((2, 150, 20))                       # cached: the kept positions, then the window
    assert rec == [[0, 20, 25, 99, 20, 5, 51, 0]]
    assert where == [[2, j] for j in (0, 1, 2, 3, 4, *range(51, 170))]
    rec, where = pieces((2, 102, 20))                       # the window still reaches some of them
    assert rec == [[0, 20, 23, 99, 20, 5, 3, 0]] and where == [[2, j] for j in (0, 1, 2, *range(3, 122))]
    rec, where = pieces((2, 60, 20))                        # all of them
    assert rec == [[0, 20, 20, 60, 20, 0, 0, 0]] and where == [[2, j] for j in range(80)]


def test_window_pieces_leave_the_rest_of_the_batch_alone():
    """Entries of a recurrence's plan beside pieces of a window."""
    scan = R.ScanPlan(4, True)
    b = R.RaggedBatch([R.Entry(0, 0, [0] * 30), R.Entry(1, 5, [0])], "cpu", plans=[R.AttnPlan(None, True, 100), scan])
    assert b.scan(scan)[0] == 1 and b.scan(scan)[5].tolist() == [1] and b.positions.numel() == 31 + 2

"""Sapasun on CPU in fp32: every mechanism and the whole serving path (step, cache, state, engine,
scheduler, command line, trace runner) against the plain implementation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_sapasun as plain
import sapasun_cases as cases
from coeus_b200.foundation.error import Error
from coeus_b200.infer.engine import make_engine
from coeus_b200.infer.scheduler import ContinuousBatcher
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


@pytest.mark.parametrize("kind", ["odd", "delta", "attn"])
@pytest.mark.parametrize("check", cases.MODEL_CHECKS, ids=lambda c: c.__name__[6:])
def test_model(kind, check):
    check(bench(kind))


def test_plain_chunk_counts_from_the_sequence_start():
    seen = [[j for j in range(i + 1) if plain.chunk_visible(i, j, 3)] for i in range(7)]
    assert seen == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]


def test_directory_round_trip_and_registry(tmp_path):
    b = bench("odd")
    registry.save_dir(b.lm, str(tmp_path))
    config = registry.read_config(str(tmp_path))
    assert registry.resolve(config).name == "Sapasun" and "Sapasun" in registry.architectures()
    lm = registry.load_dir(str(tmp_path), device="cpu", dtype=torch.float32)
    assert lm.cfg == b.cfg and lm.num_parameters() == b.lm.num_parameters()
    w = b.w
    got = lm.state_dict()
    assert set(got) == set(w)
    for n in w:
        assert torch.equal(got[n].float(), w[n].float()), n
    with pytest.raises(Error):
        registry.resolve({"architecture": "no such design"})
    with pytest.raises(Error):
        registry.load_dir(str(tmp_path), device="cpu", training=True)
    bad = {k: v for k, v in w.items() if k != "l2.mix.sink"}
    with pytest.raises(Error):
        H.load_hybrid(bad, config, device="cpu")
    with pytest.raises(Error):
        H.load_hybrid({**w, "l2.mix.sink": torch.zeros(5)}, config, device="cpu")


def test_config_is_checked():
    j = H.config_to_json(cases.config("odd"))
    shapes = H.tensor_shapes(cases.config("odd"))
    assert H.config_from_json(j, shapes) == cases.config("odd")

    def broken(edit):
        c = json.loads(json.dumps(j))
        edit(c)
        with pytest.raises(Error):
            H.config_from_json(c, shapes)
    broken(lambda c: c["layers"][0].update(type="other"))
    broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda c: c["layers"][1]["mixer"].update(v_mix=True))    # other value sizes than layer 2
    broken(lambda c: c["layers"][1]["mixer"].update(dim=400))


def test_step_refuses_wrong_input():
    eng = bench("odd").engine(2, max_len=128)
    for entries in ([R.Entry(0, 3, [1])],                              # starts past the slot's tokens
                    [R.Entry(0, 0, [1]), R.Entry(0, 0, [2])],          # one slot twice
                    [R.Entry(0, 0, [bench("odd").cfg.vocab_size])],    # unknown token
                    [R.Entry(0, 0, [1] * 129)]):                       # more than a slot may hold
        with pytest.raises(Error):
            eng.step(entries)
    assert eng.step([R.Entry(0, 0, [1, 2])]) is None                   # nothing wanted


def test_batcher_waits_for_pages_and_fails_the_impossible():
    b = bench("delta")
    eng = make_engine(b.lm, max_batch=3)
    cb = ContinuousBatcher(eng, max_seqs=3, max_len=192)
    eng.open_slots(3, 192, num_pages=2)           # fewer pages than the slots could use
    ok = [cb.submit(cases.tokens(b.cfg, 70, s), 3) for s in (1, 2)]    # two pages each: one at a time
    big = cb.submit(cases.tokens(b.cfg, 150, 3), 3)
    done = {}
    while cb.pending():
        for r in cb.step():
            done[r.id] = r
    assert done[big].error is not None
    for rid in ok:
        assert done[rid].error is None
        cases.agrees(b, done[rid].prompt, done[rid].output)
    with pytest.raises(Error):
        ContinuousBatcher(make_engine(b.lm), max_seqs=2, prefix_cache=True)


def test_serving_loop():
    from coeus_b200.serve import ServingLoop
    b = bench("odd")
    loop = ServingLoop(b.lm, max_seqs=2, max_len=96)
    try:
        prompts = [cases.tokens(b.cfg, n, n) for n in (3, 30, 12)]
        futs = [loop.submit(p, 5) for p in prompts]
        for p, f in zip(prompts, futs):
            out = f.result(timeout=60)
            assert len(out) == 5
            cases.agrees(b, p, out)
    finally:
        loop.close()


def _run(args, **kw):
    return subprocess.run([sys.executable, *args], capture_output=True, text=True, timeout=300,
                          cwd=ROOT, **kw)


def test_command_line(tmp_path):
    b = bench("attn")
    registry.save_dir(b.lm, str(tmp_path))
    prompt = cases.tokens(b.cfg, 9, 4)
    r = _run(["-m", "coeus_b200", "generate", "--device=cpu", f"--weights={tmp_path}",
              "--prompt_ids=" + ",".join(map(str, prompt)), "--max_tokens=6"])
    assert r.returncode == 0, r.stderr
    out = json.loads(r.stdout.strip().splitlines()[-1])
    cases.agrees(b, prompt, out["token_ids"])
    r = _run(["-m", "coeus_b200", "info", f"--weights={tmp_path}"])
    assert json.loads(r.stdout.strip().splitlines()[-1])["architecture"] == "Sapasun"


def test_trace_runner(tmp_path):
    """The program as a user calls it: steps on standard input, logits in files, slots and pages
    used again, one request left out for a step."""
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


def test_other_decoders_take_steps_too():
    """The decoder with its own slot kernels replays a trace through the same runner interface."""
    from coeus_b200.infer.trace import TraceRunner
    from coeus_b200.models.config import DecoderConfig
    from coeus_b200.models.decoder import DecoderLM
    m = DecoderLM(DecoderConfig(hidden_dim=32, num_layers=2, num_heads=2, intermediate_dim=64,
                                vocab_size=96, max_seq_len=160, use_bias=False, activation="swiglu",
                                norm="rmsnorm", pos="rope"), "cpu", dtype=torch.float32,
                  training=False)
    run = TraceRunner(make_engine(m, max_batch=4), 256)
    ids = [[3, 5, 7, 11, 13], [17, 19, 23]]
    got = run.step([{"id": "a", "tokens": ids[0][:3], "want": [2]},
                    {"id": "b", "tokens": ids[1], "want": [0, 2]}], ["b"])
    more = run.step([{"id": "a", "tokens": ids[0][3:], "want": [1]}], ["a"])
    ref = [m.forward_logits(torch.tensor(x)[None], last_only=True)[0, :96].float()
           for x in (ids[0][:3], ids[1][:1], ids[1], ids[0])]
    for a, z in zip([*got, *more], ref):
        assert (torch.from_numpy(a) - z).abs().max() < 1e-4

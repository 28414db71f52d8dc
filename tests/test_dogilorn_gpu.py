"""Dogilorn on the GPU, in bf16 and in fp32: the kernels one mechanism at a time and the serving path
against the plain implementation."""
import pytest
import torch

import dogilorn_cases as cases
from coeus_b200.ops import _lib
from coeus_b200.ops import ragged as R

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
_benches = {}


def bench(kind, dtype):
    if (kind, dtype) not in _benches:
        _benches[kind, dtype] = cases.Bench(kind, "cuda", dtype)
    return _benches[kind, dtype]


@pytest.fixture(autouse=True)
def no_kernel_status():
    yield
    _lib.check_status(torch.device("cuda", 0))


@pytest.mark.parametrize("dtype", DTYPES, ids=["fp32", "bf16"])
@pytest.mark.parametrize("check", cases.MECHANISM_CHECKS, ids=lambda c: c.__name__[6:])
def test_mechanism(check, dtype):
    check("cuda", dtype, 2e-5 if dtype == torch.float32 else 0.012)


@pytest.mark.parametrize("dtype", DTYPES, ids=["fp32", "bf16"])
@pytest.mark.parametrize("kind", ["odd", "wide", "large"])
@pytest.mark.parametrize("check", cases.MODEL_CHECKS, ids=lambda c: c.__name__[6:])
def test_model(kind, check, dtype):
    check(bench(kind, dtype))


@pytest.mark.parametrize("n", [2, 20])
def test_graph_and_plain_steps_agree(n):
    """Decoding replayed from a graph gives what the same step gives launched kernel by kernel, also
    when the slots of the batch change between replays; few rows and enough to sort them by expert."""
    b = bench("wide", torch.bfloat16)
    ids = [cases.tokens(b.cfg, 40, s) for s in range(2 * n)]
    got = []
    for graph in (True, False):
        eng = b.engine(2 * n, max_len=64, use_graph=graph)
        eng.step([R.Entry(i, 0, s[:10], []) for i, s in enumerate(ids)])
        rows = []
        for k in range(20):
            slots = [(3 * k + i) % (2 * n) for i in range(n)][::1 - 2 * (k % 2)]
            rows.append(eng.step([R.Entry(i, eng.cache.length(i), [ids[i][eng.cache.length(i)]], [0])
                                  for i in slots]).clone())
        got.append(torch.cat(rows))
    # the graph's bound on the context may split a row's keys differently: rounding only
    err = (got[0] - got[1]).square().mean(-1).sqrt() / got[1].std()
    assert float(err.max()) < 1e-2

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


@pytest.mark.parametrize("dim, window, keep", [(128, 200, 4), (128, 1024, 130), (64, 1, 3), (64, 300, 4)])
def test_long_prompts_with_many_pieces(dim, window, keep):
    """More query tiles than the GPU has SMs, so that every CTA works on several and the tiles of a pair get out
    of step; three sequences, one of which continues behind cached keys."""
    spec = cases.A(16, 2, dim, dim, dim ** -0.5, 0, 1.0, window, keep)
    plan = R.AttnPlan(None, True, window, keep=keep)
    lens, start = (2100, 1500, 900), (0, 0, 700)
    entries = [R.Entry(i, p, [0] * n) for i, (n, p) in enumerate(zip(lens, start))]
    b = R.RaggedBatch(entries, torch.device("cuda"), plans=[plan])
    g = torch.Generator(device="cuda").manual_seed(dim + window)
    pages = [(n + p + 63) // 64 for n, p in zip(lens, start)]
    table = torch.zeros((3, max(pages)), dtype=torch.int32, device="cuda")
    order = torch.randperm(sum(pages), generator=torch.Generator().manual_seed(1)).int().cuda()
    k_cache, v_cache = (torch.randn((sum(pages), 64, 2, dim), generator=g, device="cuda").bfloat16() for _ in "kv")
    q = 4.0 * torch.randn((b.T, 16, dim), generator=g, device="cuda").bfloat16()
    k_rows, v_rows = (torch.full((b.kv_rows(plan), 2, dim), float("nan"), device="cuda").bfloat16() for _ in "kv")
    wants, at = [], 0
    for i, (n, p) in enumerate(zip(lens, start)):
        own = order[sum(pages[:i]):sum(pages[:i + 1])]
        table[i, :pages[i]] = own
        k, v = (c[own.long()].flatten(0, 1)[:n + p] for c in (k_cache, v_cache))
        k_rows[at:at + n], v_rows[at:at + n] = k[p:], v[p:]
        full = torch.zeros((n + p, 16, dim), device="cuda").double()
        full[p:] = q[at:at + n].double()
        wants.append(cases.plain.attend(full, k.double(), v.double(), spec.scale, torch.ones(16), window, keep)[p:])
        at += n
    want = torch.cat(wants).flatten(1)
    for _ in range(5):
        out = torch.full((b.T, 16 * dim), 7.0, device="cuda").bfloat16()
        R.ragged_attention(q, k_cache, v_cache, table, b, 16, 2, dim, dim, spec.scale, out, window=window, keep=keep,
                           sink=torch.zeros(16, device="cuda"), k_rows=k_rows, v_rows=v_rows, plan=plan)
        err = (out.double() - want).abs().amax(1) / want.abs().max()
        assert float(err.max()) < 0.02, (int(err.argmax()), float(err.max()))


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

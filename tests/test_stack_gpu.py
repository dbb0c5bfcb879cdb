"""The serving decoder of small Lederax models on a GPU (kernels in fp32 and bf16) against the plain implementation:
whole prompts, portions, mixed batches, decoding through the engine with CUDA graphs, long decoding across pages."""
import pytest
import torch

from cosmos_b200 import ops
from tests import oracle_lederax as orc
from tests import stack_cases as cases
from tests import stack_checks as checks

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 2e-5, BF16: 6e-2}   # bf16: rounding of weights' products and activations through peaky layers


@pytest.fixture(autouse=True)
def _status_clean():
    assert ops.load_extension()
    yield
    torch.cuda.synchronize()
    ops.check_status()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_whole_prompt_and_residual_stream(tmp_path, name, dtype):
    checks.whole_prompt_and_layers(tmp_path, name, dtype, "cuda", TOL[dtype], page_size=8)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name,page,n", [("mixed", 5, 61), ("late_mix", 8, 61), ("tc", 8, 150), ("tc", 32, 150)])
def test_portions_equal_the_whole_prompt(tmp_path, name, page, n, dtype):
    checks.portions_and_token_by_token(tmp_path, name, dtype, "cuda", TOL[dtype], n=n, page_size=page)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "tc"])
def test_batches_of_unequal_requests_equal_each_alone(tmp_path, name, dtype):
    checks.mixed_batches(tmp_path, name, dtype, "cuda", TOL[dtype], page_size=16)


@pytest.mark.parametrize("dtype,slack", [(F32, 1e-4), (BF16, 0.2)])
@pytest.mark.parametrize("name,graph", [("mixed", True), ("tc", True), ("tc", False)])
def test_greedy_generation_through_the_engine(tmp_path, name, graph, dtype, slack):
    checks.greedy_generation(tmp_path, name, dtype, "cuda", slack, graph, page_size=8)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding_over_many_windows_and_pages(tmp_path, dtype):
    cfg, t, dec = checks.setup(tmp_path, "tc", dtype, "cuda", page_size=16)
    ids = cases.tokens(cfg, 330, 8)
    want = orc.forward(cfg, t, ids)
    got = cases.feed(dec, 0, ids, [30] + [1] * 300)
    e = cases.error(got, want)
    assert e < TOL[dtype], f"{e:.3g}"


def test_results_do_not_depend_on_pages_left_by_others(tmp_path):
    """The same request on fresh pages, on pages that others have used, and next to others: bit-equal logits per path."""
    cfg, t, dec = checks.setup(tmp_path, "tc", BF16, "cuda", page_size=8)
    ids = cases.tokens(cfg, 70, 1)
    first = cases.feed(dec, 0, ids, [33])
    for k in range(1, 4):
        cases.feed(dec, k, cases.tokens(cfg, 90, k), [41])
    dec.cache.release(0)
    dec.cache.release(2)
    again = cases.feed(dec, 9, ids, [33])
    assert torch.equal(first, again)

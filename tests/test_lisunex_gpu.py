"""The Lisunex design on the sm_100a kernels, in bf16 and in the 32-bit mode."""
import pytest
import torch

import lisunex_cases as cases
from kotodama_b200.ops import get_ops
from kotodama_b200.ops.cuda import KernelError

pytestmark = pytest.mark.gpu
DTYPES = [torch.bfloat16, torch.float32]


@pytest.mark.parametrize("dtype", DTYPES)
def test_row_operations(dtype):
    cases.check_row_ops(get_ops("cuda"), "cuda", dtype)
    cases.check_rotary(get_ops("cuda"), "cuda", dtype)
    get_ops("cuda").check_status()


class _PlainContext:
    """The 32-bit mode reads the paged cache in every pass: it has no packed attention."""

    def __init__(self, ops):
        self.paged_attention = ops.paged_attention


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", cases.ATTENTION_CASES, ids=str)
def test_attention_at_chunk_borders_and_far_keys(case, dtype):
    ops = get_ops("cuda")
    if dtype == torch.float32:
        case = case[:-1]
    cases.check_attention(ops if dtype == torch.bfloat16 else _PlainContext(ops), "cuda", dtype, *case)
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", cases.DELTA_CASES, ids=str)
def test_delta_rule(case, dtype):
    cases.check_delta(get_ops("cuda"), "cuda", dtype, *case)
    get_ops("cuda").check_status()


@pytest.mark.parametrize("case", [(2, 1, 64, 64, 4, [200, 64]), (3, 3, 128, 192, 4, [65, 1, 300]), (4, 1, 104, 40, 2, [128, 127])], ids=str)
def test_chunks_and_single_tokens_agree(case):
    """The chunked form against the token-by-token kernel on the same bf16 inputs: what is left is the rounding of the convolutions."""
    ops = get_ops("cuda")
    H, G, d, dv, taps, lens = case
    parts, w = cases.delta_case(H, G, d, dv, taps, lens, 3, dtype=torch.bfloat16)
    sequences = [(sum(lens[:i]), sum(lens[:i + 1])) for i in range(len(lens))]
    args = (ops, "cuda", parts, w, H, G, d, dv, 1e-5, sequences)
    slots = list(range(len(lens)))
    whole, s1 = cases.run_delta(*args, [lens], slots)
    short = type(ops).delta_short
    try:
        ops.delta_short = 10 ** 9
        walked, s2 = cases.run_delta(*args, [lens], slots)
    finally:
        ops.delta_short = short
    for a, b in zip(whole, walked):
        assert float(((a - b).norm(dim=-1) / b.norm(dim=-1)).max()) < 0.02
    n = len(lens)
    assert float((s1[:n, ..., :dv] - s2[:n, ..., :dv]).norm() / s2[:n, ..., :dv].norm()) < 3e-3
    ops.check_status()


def test_operands_that_do_not_belong_together_are_refused():
    ops = get_ops("cuda")
    parts, w = cases.delta_case(1, 1, 64, 64, 2, [40], dtype=torch.bfloat16)
    rows = cases.join(parts).cuda()
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    state, ring = torch.zeros(4, 1, 64, 64, device="cuda"), torch.zeros(4, 1, 1, 192, device="cuda", dtype=torch.bfloat16)
    call = lambda slots, cu, ctx: ops.delta_rule(rows, 1, 1, 64, 64, *(w[x].cuda() for x in ("conv", "a_log", "dt", "norm")), 1e-5, state, ring, slots, cu, ctx, 40)
    with pytest.raises(KernelError):
        call(i32([0, 1, 2]), i32([0, 40]), i32([40]))
    with pytest.raises(KernelError):
        call(i32([0]), None, i32([1]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype):
    cases.check_portions(name, "cuda", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_and_slots_used_again(dtype):
    for name in ("odd", "fit"):
        cases.check_batches(name, "cuda", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_behind_the_chunk_are_given_back(dtype):
    cases.check_pages_behind_the_chunk("fit", "cuda", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    cases.check_long_decoding("fit", "cuda", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(dtype):
    cases.check_generation("odd", "cuda", dtype)
    cases.check_generation("fit", "cuda", dtype)


def test_decode_graphs_and_plain_launches_agree():
    """Capturing a graph (which runs the step once to warm up) must not advance the recurrent states."""
    cfg = cases.CONFIGS["fit"]
    model = cases.weights(cfg, 9)
    outs = []
    for graphs in (True, False):
        eng = cases.engine(model, "cuda", torch.bfloat16)
        eng.use_cuda_graphs = graphs
        outs.append(cases.feed(eng, eng.open(), cases.tokens(cfg, 60, 2), [20, 1]))
    assert float((outs[0] - outs[1]).abs().max()) < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
def test_kernels_write_inside_their_tensors(dtype):
    """Canary bands around every allocation: prompts, portions, decoding at ragged sizes."""
    from kotodama_b200.utils.guard import GuardRegions
    with GuardRegions() as g:
        for name in ("odd", "fit", "wide"):
            cfg = cases.CONFIGS[name]
            eng = cases.engine(cases.weights(cfg, 4), "cuda", dtype, max_ctx=400)
            eng.use_cuda_graphs = False
            s, t = eng.open(), eng.open()
            toks = cases.tokens(cfg, 340, 3)
            eng.feed([(s, toks[:301], [0, 300]), (t, toks[:7], [6])])
            eng.feed([(s, toks[301:304], [2]), (t, toks[7:27], [])])
            for i in range(5):
                eng.feed([(s, [toks[304 + i]], [0]), (t, [toks[27 + i]], [0])])
        torch.cuda.synchronize()
        g.assert_clean()
    get_ops("cuda").check_status()

"""The Vunitar design on the sm_100a kernels, in bf16 and in the 32-bit mode."""
import pytest
import torch

import vunitar_cases as cases
from kotodama_b200.ops import get_ops
from kotodama_b200.ops.reference import TORCH_OPS

pytestmark = pytest.mark.gpu
DTYPES = [torch.bfloat16, torch.float32]


@pytest.mark.parametrize("dtype", DTYPES)
def test_row_operations(dtype):
    cases.check_ops(get_ops("cuda"), "cuda", dtype)
    get_ops("cuda").check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_routing_and_experts(dtype):
    cases.check_experts(get_ops("cuda"), "cuda", dtype)
    cases.check_experts(get_ops("cuda"), "cuda", dtype, N=300)       # router as a product, 128-row expert tiles
    get_ops("cuda").check_status()


class _Fp32Context:
    """The 32-bit mode has no packed attention of its own: far keys are checked on the latent form."""

    def __init__(self, ops):
        self.latent_attention, self.attention_context = ops.latent_attention, TORCH_OPS.attention_context


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_and_the_causal_edge(dtype):
    ops = get_ops("cuda")
    cases.check_far_keys(ops if dtype == torch.bfloat16 else _Fp32Context(ops), "cuda", dtype)
    cases.check_far_keys(ops if dtype == torch.bfloat16 else _Fp32Context(ops), "cuda", dtype, R=384, H=18)
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype):
    cases.check_portions(name, "cuda", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_and_reused_pages(dtype):
    for name in ("odd", "wide"):
        cases.check_batches(name, "cuda", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    cases.check_long_decoding("plain", "cuda", dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(dtype):
    cases.check_generation("odd", "cuda", dtype)
    cases.check_generation("plain", "cuda", dtype)


@pytest.mark.parametrize("H,R,lens,news", [(16, 512, [300, 40, 1, 1000], [1] * 4), (24, 256, [300, 77], [3, 5]), (128, 512, [129], [1]),
                                           (5, 640, [2000, 15, 16], [2, 1, 16]), (40, 128, [63] * 70, [1] * 70), (8, 1024, [200], [1])])
def test_latent_attention_against_fp32(H, R, lens, news):
    """Unequal contexts and portions in one launch; work pieces that cut sequences; a latent too large for the ring."""
    ops = get_ops("cuda")
    g = torch.Generator().manual_seed(H)
    mp = max((c + 15) // 16 for c in lens) + 1
    P = len(lens) * mp + 3
    pages = torch.randn(P, R // 64, 16, 64, generator=g).bfloat16().cuda()
    table = torch.randperm(P, generator=g)[: len(lens) * mp].int().view(len(lens), mp).contiguous().cuda()
    cu = torch.tensor([0] + list(torch.tensor(news).cumsum(0)), dtype=torch.int32).cuda()
    q = torch.randn(sum(news), H, R, generator=g).bfloat16().cuda()
    ctx = torch.tensor(lens, dtype=torch.int32).cuda()
    out = ops.latent_attention(q, pages, table, ctx, None if max(news) == 1 else cu, max(news), max(lens), 0.1)
    ops.check_status()
    want = TORCH_OPS.latent_attention(q.float(), pages.float(), table, ctx, cu, max(news), max(lens), 0.1)
    assert float(((out.float() - want).norm(dim=-1) / want.norm(dim=-1)).max()) < 0.01


@pytest.mark.parametrize("rows", [[5], [0, 3, 0, 0, 129, 1, 0], [128, 256, 127], [33] * 40, [0, 0, 1]])
@pytest.mark.parametrize("N,K", [(40, 24), (264, 328), (512, 64)])
def test_grouped_product_against_fp32(rows, N, K):
    """Empty groups, groups of one row, groups that end on and beside the tile; both tile heights; column and K tails."""
    ops = get_ops("cuda")
    g = torch.Generator().manual_seed(N + len(rows))
    A = sum(rows)
    a = torch.randn(A, K, generator=g).bfloat16().cuda()
    w = (torch.randn(len(rows), N, K, generator=g) * K ** -0.5).bfloat16().cuda()
    off = torch.tensor([0] + list(torch.tensor(rows).cumsum(0)), dtype=torch.int32).cuda()
    for kind in (None, "gelu", "relu2"):
        out = ops._grouped(a, w, off, kind)
        ops.check_status()
        want = torch.cat([a[off[i]:off[i + 1]].float() @ w[i].float().t() for i in range(len(rows))])
        want = TORCH_OPS.activate(want, kind) if kind else want
        assert float((out.float() - want).abs().max()) < 0.03 * (1 + float(want.abs().max()) * 0.3), (kind, rows)


def test_fp32_products_are_true_fp32():
    """No reduced-precision matrix mode: the error is fp32 rounding, not the 1e-3 of a truncated mantissa."""
    ops = get_ops("cuda")
    g = torch.Generator().manual_seed(0)
    a, b = torch.randn(70, 515, generator=g), torch.randn(131, 515, generator=g)
    want = a.double() @ b.double().t()
    assert float((ops.gemm_nt(a.cuda(), b.cuda()).double().cpu() - want).abs().max()) < 2e-4
    res = torch.randn(70, 131, generator=g)
    got = ops.gemm_nt(a.cuda(), b.cuda(), residual=res.cuda())
    assert float((got.double().cpu() - want - res.double()).abs().max()) < 2e-4


def test_decode_graphs_and_plain_launches_agree():
    cfg = cases.CONFIGS["wide"]
    model = cases.weights(cfg, 9)
    outs = []
    for graphs in (True, False):
        eng = cases.engine(model, "cuda", torch.bfloat16)
        eng.use_cuda_graphs = graphs
        s = eng.open()
        outs.append(cases.feed(eng, s, cases.tokens(cfg, 60, 2), [20, 1]))
    assert float((outs[0] - outs[1]).abs().max()) < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
def test_kernels_write_inside_their_tensors(dtype):
    """Canary bands around every allocation: prompts, portions, decoding and generation at ragged sizes."""
    from kotodama_b200.utils.guard import GuardRegions
    with GuardRegions() as g:
        for name in ("odd", "wide"):
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

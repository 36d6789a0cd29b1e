"""Small Vunitar configurations and the checks that run on both back ends (CPU in fp32, CUDA in bf16 and fp32), against
the plain implementation in ``vunitar_oracle.py``."""
import torch

import vunitar_oracle as oracle
from kotodama_b200.models.vunitar import VunitarConfig, VunitarModel
from kotodama_b200.serve.engine import SamplingParams, ServingEngine


def mixer(heads, dim, vdim, rank, scale):
    return dict(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, scale=scale)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, shared=None, groups=None, scale=1.0):
    d = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))
    if groups:
        d["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared:
        d["shared"] = dict(ff=shared)
    return d


def config(vocab, width, layers, bigram=None, softcap=None, eps=1e-5):
    d = dict(architecture="Vunitar", vocab=vocab, width=width, norm=dict(eps=eps),
             layers=[dict(type="latent_attention", mixer=m, mlp=f) for m, f in layers])
    if bigram:
        d["embedding"] = dict(bigram=dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2]))
    if softcap:
        d["logit_softcap"] = softcap
    return d


CONFIGS = {
    # nothing is a multiple of eight; every kind of feed-forward, the expert layer first; sizes differ from layer to layer
    "odd": config(101, 84, [(mixer(3, 20, 28, 36, 0.31), moe(6, 2, 20, 27, (3, 2), 1.7)), (mixer(5, 12, 9, 50, 0.2), None),
                            (mixer(1, 33, 17, 20, 0.15), dense(75))], (37, 11, 5), 9.0, 3e-4),
    # no bigram, no soft-cap, no shared expert, no groups; heads of 80 on the 128-wide tile
    "plain": config(300, 128, [(mixer(4, 80, 48, 160, 0.12), dense(256)), (mixer(4, 80, 48, 160, 0.12), moe(8, 3, 40))]),
    # heads wider than the flash kernel takes; one group kept, all experts of it chosen; value wider than key
    "wide": config(200, 96, [(mixer(2, 136, 152, 64, 0.09), moe(12, 4, 24, 40, (3, 1), 2.0)), (mixer(20, 24, 64, 272, 0.2), dense(64))],
                   (64, 3, 7), 25.0),
    # one of everything
    "one": config(64, 32, [(mixer(1, 16, 16, 16, 0.25), moe(1, 1, 16, 16, (1, 1)))], (1, 1, 1), 5.0),
}


def weights(cfg, seed=0):
    """Random bf16 weights with sharp attention (queries scaled up) and well separated router scores."""
    m = VunitarModel.random_init(VunitarConfig.from_dict(cfg), seed)
    for name, t in m.weights.items():
        if name.endswith("mix.q"):
            t.mul_(2.0)
        elif name.endswith("mlp.router"):
            t.mul_(3.0)
    return m


class Expected(torch.Tensor):
    """Logits of the plain implementation; ``sure``: rows whose routers decided by more than rounding can turn."""


def oracle_logits(cfg, model, tokens):
    margins = []
    out = oracle.forward(cfg, {k: v.double() for k, v in model.weights.items()}, tokens, margins_out=margins)
    out = torch.Tensor._make_subclass(Expected, out)
    out.sure = (torch.tensor(margins).amin(0) > 0.25) if margins else torch.ones(len(tokens), dtype=torch.bool)
    return out


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(model, device, dtype, **kw):
    return ServingEngine(model, device=device, dtype=dtype, **{"max_batch": 4, "max_ctx": 704, **kw})


def row_errors(got, want):
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def assert_close(got, want, dtype, what="", rows=None):
    """fp32: every row.  bf16: most of the rows whose routing is not a close call (a token whose expert did change is a
    key of the later ones).  ``rows`` of the plain logits, default the first ``len(got)``."""
    rows = list(range(got.shape[0])) if rows is None else rows
    plain = want.as_subclass(torch.Tensor)
    e = row_errors(got, plain[rows])
    assert torch.isfinite(e).all(), what
    if dtype == torch.float32:
        assert float(e.max()) < 1e-4, (what, float(e.max()))
        return
    e = e[want.sure[rows]]
    if e.numel():
        over = int((e > 0.05).sum())
        assert over <= max(1, 0.2 * e.numel()) and float(e.max()) < 0.5 and float(e.median()) < 0.025, (
            what, float(e.median()), float(e.max()), over, e.numel())


def feed(eng, seq, toks, cuts):
    """Feeds ``toks`` in portions of the given sizes (the last size repeats); returns all logits."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(eng.feed([(seq, toks[at:at + n], list(range(n)))])[0])
        at, k = at + n, k + 1
    return torch.cat(out)


def check_portions(name, device, dtype, lengths=(1, 2, 50, 300)):
    """Whole prompts, token by token, and portions down to two tokens give the plain implementation's logits."""
    cfg = CONFIGS[name]
    model = weights(cfg)
    eng = engine(model, device, dtype)
    for n in lengths:
        toks = tokens(cfg, n, n)
        want = oracle_logits(cfg, model, toks)
        ways = {"whole": [n], "portions": [33, 2, 17, 1, 64, 3, 16], "twos": [max(1, n - 30), 2], "decode": [max(1, n - 40), 1]}
        first = None
        for way, cuts in ways.items():
            seq = eng.open()
            got = feed(eng, seq, toks, cuts)
            assert_close(got, want, dtype, (name, n, way))
            # whatever the portions, the same numbers up to rounding (and to routers that decide on it)
            first = got if first is None else first
            e = row_errors(got, first.double())[want.sure]
            limit, few = (0.05, max(1, 0.1 * n)) if dtype == torch.bfloat16 else (2e-5, 0)
            assert int((e > limit).sum()) <= few, (name, n, way, float(e.max()))
            eng.close(seq)
    assert sorted(eng.cache.free) == list(range(eng.cache.num_pages))
    if hasattr(eng.ops, "check_status"):
        eng.ops.check_status()


def check_batches(name, device, dtype):
    """Sequences of unequal lengths in one pass, prompts beside single tokens, equal each alone."""
    cfg = CONFIGS[name]
    model = weights(cfg, 1)
    eng = engine(model, device, dtype)
    lens = [40, 7, 129, 18]
    toks = [tokens(cfg, n, 100 + n) for n in lens]
    want = [oracle_logits(cfg, model, t) for t in toks]
    seqs = [eng.open() for _ in lens]
    at = [0] * len(lens)
    got = [[] for _ in lens]
    plan = [(20, 3, 100, 0), (1, 1, 1, 16), (5, 1, 20, 1), (1, 1, 1, 1), (1, 1, 7, 0), (12, 0, 0, 0)]
    for step in plan:
        entries = [(i, min(n, lens[i] - at[i])) for i, n in enumerate(step) if n and at[i] < lens[i]]
        outs = eng.feed([(seqs[i], toks[i][at[i]:at[i] + n], list(range(n))) for i, n in entries])
        for (i, n), o in zip(entries, outs):
            got[i].append(o)
            at[i] += n
    for i, n in enumerate(lens):
        assert_close(torch.cat(got[i]), want[i], dtype, (name, "batch", i))
        assert at[i] == n
    # what was freed is used again, by other sequences in another order
    for s in (seqs[2], seqs[0]):
        eng.close(s)
    again = eng.open()
    t = tokens(cfg, 200, 7)
    assert_close(feed(eng, again, t, [60, 2, 90, 1]), oracle_logits(cfg, model, t), dtype, (name, "reused pages"))


def check_long_decoding(name, device, dtype, n=420):
    cfg = CONFIGS[name]
    model = weights(cfg, 2)
    eng = engine(model, device, dtype)
    toks = tokens(cfg, n, 5)
    seq = eng.open()
    assert_close(feed(eng, seq, toks, [3, 1]), oracle_logits(cfg, model, toks), dtype, (name, "long decoding"))


def greedy(cfg, model, prompt, n):
    toks, out = list(prompt), []
    for _ in range(n):
        out.append(int(oracle_logits(cfg, model, toks)[-1].argmax()))
        toks.append(out[-1])
    return out


def check_generation(name, device, dtype):
    """Greedy generation through the scheduler: more prompts than batch slots, prompts in portions or whole."""
    cfg = CONFIGS[name]
    model = weights(cfg, 3)
    prompts = [tokens(cfg, n, 30 + n) for n in (5, 41, 1, 18, 33)]
    want = [greedy(cfg, model, p, 8) for p in prompts]
    for portion in (0, 2, 16, 24):
        eng = engine(model, device, dtype, max_batch=3, max_ctx=64, prefill_portion=portion)
        got = eng.generate(prompts, SamplingParams(max_new_tokens=8, temperature=0.0))
        if dtype == torch.float32:
            assert got == want, (name, portion)
        else:                       # rounding may turn a near-tie, after which the texts part
            assert sum(g[:3] == w[:3] for g, w in zip(got, want)) >= 4, (name, portion, got, want)
        assert len(eng.cache.free) == eng.cache.num_pages


# ---------------------------------------------------------------------------------- mechanisms alone
def pages_for(rows, page_ids, block):
    """Cache pages holding ``rows`` in the given page order."""
    n, R = rows.shape
    pages = torch.zeros(max(page_ids) + 1, R // block, 16, block, dtype=rows.dtype, device=rows.device)
    for i in range(n):
        pages[page_ids[i // 16], :, i % 16] = rows[i].view(R // block, block)
    return pages


def check_far_keys(ops, device, dtype, R=128, H=3, ctx=700):
    """One key per head stands out; it must be found wherever it is, and must not be seen from just in front of it.  The
    queries are decoded alone, in portions, and (expanded keys) in the packed form."""
    g = torch.Generator().manual_seed(0)
    c = torch.randn(ctx, R, generator=g)
    c = c / c.norm(dim=-1, keepdim=True)
    ids = torch.randperm((ctx + 15) // 16 + 3, generator=g).tolist()[: (ctx + 15) // 16]
    pages = pages_for(c.to(dtype), ids, 64 if device == "cuda" and dtype == torch.bfloat16 else R).to(device)
    crows = c.to(dtype).float()
    table = torch.tensor([ids], dtype=torch.int32, device=device)
    tol = 0.02 if dtype == torch.bfloat16 else 1e-5
    spots = [0, 1, 14, 15, 16, 17, 126, 127, 128, 129, 255, 256, 383, 384, 511, 512, 640, ctx - 2, ctx - 1]
    for n in (1, 2, 5, 16):
        for t0 in range(0, len(spots), H):
            mark = spots[t0:t0 + H] + [0] * (H - len(spots[t0:t0 + H]))
            q = torch.stack([c[m] * 60.0 for m in mark]).to(dtype).repeat(n, 1, 1).to(device)
            cu = torch.tensor([0, n], dtype=torch.int32, device=device)
            out = ops.latent_attention(q, pages, table, torch.tensor([ctx], dtype=torch.int32, device=device), cu if n > 1 else None,
                                       n, ctx, 1.0).float().cpu()
            for i in range(n):
                last = ctx - n + i
                s = (q[i].float().cpu() @ crows.t())[:, : last + 1]
                want = torch.softmax(s, -1) @ crows[: last + 1]
                assert float((out[i] - want).abs().max()) < tol, (n, i, mark)
                for h, m in enumerate(mark):
                    seen = float(out[i, h] @ c[m]) > 0.9
                    assert seen == (m <= last), (n, i, m)
    # packed queries against expanded keys: every portion size and offset meets the same key
    hd = 64
    k = torch.randn(ctx, H, hd, generator=g)
    k = k / k.norm(dim=-1, keepdim=True)
    kd = k.to(dtype).to(device)
    for n in (1, 17, 130, 257, ctx):
        for m in (0, 15, 127, 128, ctx - 129, ctx - 2, ctx - 1):
            q = (k[m] * 60.0).to(dtype).repeat(n, 1, 1).to(device)
            out = ops.attention_context(q, kd, kd, torch.tensor([0, n], dtype=torch.int32, device=device),
                                        torch.tensor([0, ctx], dtype=torch.int32, device=device), n, 1.0).float().cpu()
            last = torch.arange(ctx - n, ctx)
            dot = torch.einsum("nhd,hd->nh", out, kd[m].float().cpu())
            assert ((dot > 0.9) == (m <= last)[:, None]).all(), (n, m)


def check_ops(ops, device, dtype):
    """Row operations one by one against the plain functions."""
    g = torch.Generator().manual_seed(4)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 2e-2 if dtype == torch.bfloat16 else 2e-6
    dev = lambda t: t.to(device)
    close = lambda a, b, t=None: bool(((a.double().cpu() - b).abs() <= (t or tol) * (1 + b.abs())).all())

    # pair embedding: first tokens, wrap-around, padding of the width
    V, D, Dp = 50, 36, 40
    table, bigram = rnd(V, D).to(dtype), rnd(8, D).to(dtype)
    toks = tokens(dict(vocab=V), 30, 1)
    pad = lambda t, n: torch.cat([t, torch.zeros(*t.shape[:-1], n - t.shape[-1], dtype=t.dtype)], -1)
    prev = torch.tensor([-1] + toks[:-1], dtype=torch.int32)
    x, h = ops.embed_pairs(dev(torch.tensor(toks)), dev(prev), dev(pad(table, Dp)), dev(pad(bigram, Dp)), (7, 131, 17))
    want = oracle.embed(toks, table.double(), bigram.double(), dict(buckets=7, mul_prev=131, mul_cur=17))
    assert close(x[:, :D], want, 1e-6) and float(x[:, D:].abs().max()) == 0 and close(h[:, :D], want)

    # latent norm, cache slots, gather; a dropped slot
    R, Rp, n = 20, 24, 21
    raw, w = rnd(n, R), rnd(R)
    ids = [3, 0]
    slots = torch.tensor([ids[i // 16] * 16 + i % 16 for i in range(n)])
    slots[5] = -1
    pages = torch.zeros(5, Rp // 8, 16, 8, dtype=dtype, device=device)
    got = ops.latent_append(dev(pad(raw.to(dtype), Rp)), dev(pad(w, Rp)), R, 1e-3, pages, dev(slots))
    want = oracle.rms(raw.to(dtype).double(), w.double(), 1e-3)
    assert close(got[:, :R], want)
    cu = torch.tensor([0, n], dtype=torch.int32, device=device)
    back = ops.latent_gather(pages, dev(torch.tensor([ids], dtype=torch.int32)), cu, n).cpu()
    got[5] = 0
    assert torch.equal(back, got.cpu())

    # output norm + layer scale + residual; final norm of chosen rows
    x0, y, gn = rnd(n, D), rnd(n, D).to(dtype), rnd(D)
    x = dev(pad(x0, Dp)).clone()
    h = ops.norm_add(x, dev(pad(y, Dp)), dev(pad(gn, Dp)), D, 1e-3)
    want = x0.double() + oracle.rms(y.double(), gn.double(), 1e-3)
    assert close(x[:, :D], want, 1e-5) and close(h[:, :D], want)
    rows = torch.tensor([4, 0, 20])
    assert close(ops.norm_rows(x, dev(rows), dev(pad(gn, Dp)), D, 1e-3, dtype)[:, :D], oracle.rms(want[rows], gn.double(), 1e-3))

    # activations and the soft-cap
    u = torch.cat([torch.linspace(-9, 9, 184), torch.tensor([0.0, -0.0, 1e-4, -1e-4, 30.0, -30.0, 3.0, -3.0])]).to(dtype)
    assert close(ops.activate(dev(u), "gelu"), oracle.gelu_erf(u.double()))
    assert close(ops.activate(dev(u), "relu2"), oracle.relu_squared(u.double()))
    lg = rnd(3, 77) * 20
    assert close(ops.softcap_(dev(lg.clone()), 6.0), oracle.softcap(lg.double(), 6.0), 2e-6)

    # per-head products, both orientations
    a, wa = rnd(9, 3, 16).to(dtype), rnd(3, 16, 24).to(dtype)
    assert close(ops.head_gemm(dev(a), dev(wa), transposed=True), torch.einsum("nhk,hkm->nhm", a.double(), wa.double()))
    assert close(ops.head_gemm(dev(a), dev(wa.transpose(1, 2).contiguous())), torch.einsum("nhk,hkm->nhm", a.double(), wa.double()))


def check_experts(ops, device, dtype, N=37):
    """Routing (groups, ties in the number kept, scale, gate), the experts and their weighted sum."""
    g = torch.Generator().manual_seed(6)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 3e-2 if dtype == torch.bfloat16 else 1e-5
    for E, top, groups, ff, shared, D in ((6, 2, (3, 2), 24, True, 40), (64, 6, (8, 3), 16, False, 64), (40, 8, (1, 1), 8, True, 32),
                                          (4, 4, (2, 2), 72, False, 32), (96, 1, (96, 5), 8, True, 32)):
        h = rnd(N, D).to(dtype)
        router = rnd(E + int(shared), D).to(dtype)
        r = dict(top=top, scale=1.3, groups=dict(count=groups[0], keep=groups[1]))
        up, down = (rnd(E, ff, D) * D ** -0.5).to(dtype), (rnd(E, D, ff) * ff ** -0.5).to(dtype)
        ids, wts, gate, plan = ops.moe_route(h.to(device), router.to(device), E, top, 1.3, *groups)
        picks = oracle.route(h.double(), router[:E].double(), r)
        for i, p in enumerate(picks):
            assert ids[i].tolist() == [e for e, _ in p], (E, i)
            assert torch.allclose(wts[i].double().cpu(), torch.stack([s for _, s in p]), rtol=2e-5)
        if shared:
            assert torch.allclose(gate.double().cpu(), torch.sigmoid(h.double() @ router[E].double()), rtol=1e-4, atol=1e-6)
        ye, at = ops.moe_experts(h.to(device), ids, up.to(device), down.to(device), "gelu", plan)
        ys = rnd(N, D).to(dtype) if shared else None
        x0, gn = rnd(N, D), rnd(D)
        x = x0.clone().to(device)
        out = ops.moe_combine_norm_add(x, ye, at, wts, ys.to(device) if shared else None, gate, gn.to(device), D, 1e-4, dtype)
        y = torch.stack([sum(s * oracle.expert_ff(h[i].double()[None], up[e].double(), down[e].double())[0] for e, s in p)
                         for i, p in enumerate(picks)])
        if shared:
            y = y + torch.sigmoid(h.double() @ router[E].double())[:, None] * ys.double()
        want = x0.double() + oracle.rms(y, gn.double(), 1e-4)
        assert float((x.double().cpu() - want).abs().max()) < tol * 4, E
        assert float((out.double().cpu() - want).abs().max()) < tol * 6, E
        assert sorted(at.flatten().tolist()) == list(range(N * top))

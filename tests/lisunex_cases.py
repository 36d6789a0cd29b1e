"""Small Lisunex configurations and the checks that run on both back ends (CPU in fp32, CUDA in bf16 and fp32), against
the plain implementation in ``lisunex_oracle.py``."""
import math

import torch

import lisunex_oracle as oracle
from kotodama_b200.models.lisunex import AttentionMixer, LisunexConfig, LisunexModel, Rotary
from kotodama_b200.serve.engine import SamplingParams, ServingEngine
from vunitar_cases import feed, row_errors, tokens


def attention(heads, kv, dim, vdim, scale, rot, chunk=0, softcap=0.0, yarn=None, base=1000.0):
    r = dict(dims=rot, base=base)
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, rot=r)
    if chunk:
        m["mask"] = dict(size=chunk)
    if softcap:
        m["softcap"] = softcap
    return dict(type="attention", mixer=m)


def delta(heads, kv, dim, vdim, conv):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv))


def config(vocab, width, layers, loop=None, embedding=1.0, eps=1e-5):
    d = dict(architecture="Lisunex", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=embedding),
             layers=[dict(m, mlp=dict(kind="dense", ff=ff) if ff else None) for m, ff in layers])
    if loop:
        d["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return d


CONFIGS = {
    # nothing is a multiple of eight; sizes differ from layer to layer; a layer without chunks, cap and scaling; three passes of the loop
    "odd": config(101, 84, [(delta(6, 3, 20, 28, 4), 0), (attention(6, 2, 28, 20, 0.9, 12, 37, 7.0, (3.0, 60, 8.0, 1.0)), 75),
                            (delta(2, 1, 9, 13, 1), 50), (attention(3, 3, 33, 17, 0.5, 6), 0)], (1, 3, 3), 5.0, 3e-4),
    # heads that fit the tensor-core kernels, keys and values of different sizes, every attention layer chunked
    "fit": config(300, 128, [(delta(4, 2, 128, 64, 4), 96), (attention(4, 2, 128, 96, 0.3, 64, 48, 12.0, (4.0, 100, 16.0, 1.0)), 200),
                             (delta(4, 4, 64, 136, 3), 0), (attention(6, 1, 64, 64, 0.6, 64, 130, 200.0), 64)], (0, 2, 2), 2.0),
    # heads and taps beyond the tensor-core kernels; a cap that the scores reach; more groups than one block of heads
    "wide": config(200, 96, [(attention(22, 2, 136, 152, 0.4, 48, 65, 1.5), 100), (delta(3, 3, 160, 200, 6), 64)], (1, 2, 4)),
    # one of everything; a chunk of one token
    "one": config(64, 32, [(delta(1, 1, 8, 8, 2), 0), (attention(1, 1, 16, 16, 1.0, 2, 1, 3.0, (2.0, 8, 2.0, 1.0)), 16)], (0, 2, 1)),
}


def weights(cfg, seed=0, decays=None):
    """Random bf16 weights; ``decays``: the heads' A_log, from fast to slow."""
    m = LisunexModel.random_init(LisunexConfig.from_dict(cfg), seed)
    for name, t in m.weights.items():
        if decays and name.endswith("A_log"):
            t.copy_(torch.linspace(decays[0], decays[1], t.numel()))
    return m


def oracle_logits(cfg, model, toks):
    return oracle.forward(cfg, {k: v.double() for k, v in model.weights.items()}, toks)


def engine(model, device, dtype, **kw):
    return ServingEngine(model, device=device, dtype=dtype, **{"max_batch": 4, "max_ctx": 704, **kw})


def assert_close(got, want, dtype, what="", rows=None):
    e = row_errors(got, want if rows is None else want[rows])
    assert torch.isfinite(e).all(), what
    if dtype == torch.float32:
        assert float(e.max()) < 1e-4, (what, float(e.max()))
    else:
        assert float(e.median()) < 0.03 and float(e.max()) < 0.12, (what, float(e.median()), float(e.max()), int(e.argmax()))


def check_portions(name, device, dtype, lengths=(1, 2, 50, 200)):
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
            first = got if first is None else first
            e = row_errors(got, first.double())
            assert float(e.max()) < (0.06 if dtype == torch.bfloat16 else 2e-5), (name, n, way, float(e.max()))
            eng.close(seq)
    assert sorted(eng.cache.free) == list(range(eng.cache.num_pages))
    assert sorted(eng.cache.free_states) == list(range(eng.cache.num_states))
    if hasattr(eng.ops, "check_status"):
        eng.ops.check_status()


def check_batches(name, device, dtype):
    """Sequences of unequal lengths in one pass, prompts beside single tokens, equal each alone; what was freed (pages, state
    slots) is used again by other sequences."""
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
    for s in (seqs[2], seqs[0]):
        eng.close(s)
    for seed, cuts in ((7, [60, 2, 90, 1]), (8, [1]), (9, [2, 70])):
        again = eng.open()
        t = tokens(cfg, 90, seed)
        assert_close(feed(eng, again, t, cuts), oracle_logits(cfg, model, t), dtype, (name, "used again", seed))
        eng.close(again)


def check_long_decoding(name, device, dtype, n=330):
    """Slow and fast decays; decoding over many chunk borders."""
    cfg = CONFIGS[name]
    model = weights(cfg, 2, (-7.0, 1.0))
    toks = tokens(cfg, n, 5)
    want = oracle_logits(cfg, model, toks)
    for cuts in ([3, 1], [200, 1]):
        eng = engine(model, device, dtype)
        assert_close(feed(eng, eng.open(), toks, cuts), want, dtype, (name, "long decoding", cuts))


def check_pages_behind_the_chunk(name, device, dtype):
    """Pages in front of every visible key are given back while the sequence lives, and others may write them."""
    cfg = CONFIGS[name]
    model = weights(cfg, 6)
    sizes = [l["mixer"]["mask"]["size"] for l in cfg["layers"] if l["type"] == "attention"]
    eng = engine(model, device, dtype, num_pages=30)
    ta, tb = tokens(cfg, 260, 1), tokens(cfg, 240, 2)
    wa, wb = oracle_logits(cfg, model, ta), oracle_logits(cfg, model, tb)
    a, b = eng.open(), eng.open()
    assert_close(feed(eng, a, ta[:250], [100, 3, 147]), wa[:250], dtype, "first")
    held = eng.cache.num_pages - len(eng.cache.free)
    assert held == (250 + 15) // 16 - min(250 // s * s for s in sizes) // 16
    assert_close(feed(eng, b, tb, [90, 150]), wb, dtype, "second, in pages of the first")
    assert_close(feed(eng, a, ta[250:], [1]), wa[250:], dtype, "first again")
    eng.close(a)
    eng.close(b)
    assert sorted(eng.cache.free) == list(range(30))


def greedy(cfg, model, prompt, n):
    toks, out = list(prompt), []
    for _ in range(n):
        out.append(int(oracle_logits(cfg, model, toks)[-1].argmax()))
        toks.append(out[-1])
    return out


def check_generation(name, device, dtype):
    """Greedy generation through the scheduler: more prompts than batch and state slots, prompts in portions or whole."""
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
            assert sum(g[:3] == w[:3] for g, w in zip(got, want)) >= 3, (name, portion, got, want)
        assert len(eng.cache.free) == eng.cache.num_pages and len(eng.cache.free_states) == eng.cache.num_states


# ---------------------------------------------------------------------------------- mechanisms alone
def up8(n):
    return (n + 7) // 8 * 8


def join(parts):
    """Rows of a fused projection: every part starts at a multiple of eight columns (the gaps hold junk that nothing may read)."""
    out = []
    for p in parts:
        gap = up8(p.shape[1]) - p.shape[1]
        out += [p, torch.full((p.shape[0], gap), 77.0, dtype=p.dtype)] if gap else [p]
    return torch.cat(out, 1)


def check_row_ops(ops, device, dtype):
    g = torch.Generator().manual_seed(4)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 2e-2 if dtype == torch.bfloat16 else 3e-6
    dev = lambda t: t.to(device)
    close = lambda a, b, t=None: bool(((a.double().cpu() - b).abs() <= (t or tol) * (1 + b.abs())).all())
    pad = lambda t, n: torch.cat([t, torch.zeros(*t.shape[:-1], n - t.shape[-1], dtype=t.dtype)], -1)

    # scaled embedding
    V, D, Dp, n = 50, 36, 40, 21
    table = rnd(V, D).to(dtype)
    toks = tokens(dict(vocab=V), n, 1)
    x, _ = ops.embed_pairs(dev(torch.tensor(toks)), None, dev(pad(table, Dp)), None, (0, 0, 0), 6.5)
    assert close(x[:, :D], oracle.embed(toks, table.double(), 6.5), 1e-6) and float(x[:, D:].abs().max()) == 0

    # residual, vector of the pass and pre-norm, each present or not; chosen rows leave the residual alone
    x0, y, step, w = rnd(n, D), rnd(n, D).to(dtype), rnd(D), rnd(D)
    for use_y, use_step in ((0, 0), (1, 0), (0, 1), (1, 1)):
        x = dev(pad(x0, Dp)).clone()
        h = ops.add_norm(x, dev(pad(y, Dp)) if use_y else None, dev(pad(step, Dp)) if use_step else None, dev(pad(w, Dp)), D, 1e-3, dtype)
        want = x0.double() + (y.double() if use_y else 0) + (step.double() if use_step else 0)
        assert close(x[:, :D], want, 1e-6) and close(h[:, :D], oracle.rms(want, w.double(), 1e-3)) and h.dtype == dtype
    x, rows = dev(pad(x0, Dp)).clone(), torch.tensor([4, 0, 20])
    h = ops.add_norm(x, dev(pad(y, Dp)), None, dev(pad(w, Dp)), D, 1e-3, dtype, rows=dev(rows))
    assert torch.equal(x.cpu()[:, :D], x0) and close(h[:, :D], oracle.rms(x0.double() + y.double(), w.double(), 1e-3)[rows])

    # SwiGLU, with a bias row for all rows in the product in front of it
    a, wt, b = rnd(9, 24).to(dtype), rnd(32, 24).to(dtype), rnd(32).to(dtype)
    z = ops.gemm_nt(dev(a), dev(wt), residual=dev(b).expand(9, -1))
    want = a.double() @ wt.double().t() + b.double()
    assert close(z, want, 3e-2 if dtype == torch.bfloat16 else 1e-5)
    zc = z.double().cpu()
    assert close(ops.swiglu_fwd(z), oracle.silu(zc[:, :16]) * zc[:, 16:], 2e-2 if dtype == torch.bfloat16 else 1e-5)


def check_rotary(ops, device, dtype):
    """Angles, partial rotation, unit RMS, cache slots (one dropped), zero padding, for sizes that are and are not multiples of eight."""
    g = torch.Generator().manual_seed(5)
    tol = 2e-2 if dtype == torch.bfloat16 else 5e-6
    cases = [(3, 1, 28, 20, 12, None, 0), (4, 2, 96, 80, 32, (4.0, 128, 16.0, 1.0), 0), (2, 2, 128, 128, 128, (8.0, 64, 32.0, 1.0), 128), (5, 1, 40, 64, 40, None, 64),
             (2, 1, 16, 24, 2, (1.0, 32, 4.0, 1.0), 0), (1, 1, 7, 5, 0, None, 0), (2, 1, 136, 264, 48, None, 0)]
    for H, G, dim, vdim, rd, yarn, padded in cases:
        rot = dict(dims=rd, base=500.0)
        if yarn:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
        ours = Rotary(rd, 500.0, *(yarn or ()))
        if rd:
            freq, mult = oracle.frequencies(rot)
            assert torch.allclose(ours.frequencies(), torch.tensor(freq, dtype=torch.float64), rtol=1e-12) and abs(ours.amplitude - mult) < 1e-12
        n, first, total = 19, 230, 260
        cos, sin = ours.table(total)
        q, k, v = (torch.randn(n, h * d, generator=g).to(dtype) for h, d in ((H, dim), (G, dim), (G, vdim)))
        kd, vd = (padded, padded) if padded else (up8(dim), up8(vdim))
        kp, vp = (torch.zeros(4, G, 16, s, dtype=dtype, device=device) for s in (kd, vd))
        slots = torch.tensor([(3 if i < 16 else 1) * 16 + i % 16 for i in range(n)])
        slots[5] = -1
        pos = torch.arange(first, first + n, dtype=torch.int32)
        out = ops.head_rotary_norm(join([q, k, v]).to(device), H, G, dim, vdim, cos.to(device), sin.to(device), pos.to(device), 1e-3, kp, vp,
                                   slots.to(device), True)
        wq = oracle.rms(oracle.rotate(q.double().view(n, H, dim), rot, first), None, 1e-3)
        wk = oracle.rms(oracle.rotate(k.double().view(n, G, dim), rot, first), None, 1e-3)
        for got, want in zip(out, (wq, wk, v.double().view(n, G, vdim))):
            got = got.double().cpu()
            assert float((got[..., :want.shape[2]] - want).abs().max()) < tol * 2, (H, G, dim)
            assert got.shape[2] == want.shape[2] or float(got[..., want.shape[2]:].abs().max()) == 0
        for pages, rows in ((kp, out[1]), (vp, out[2])):
            for i in range(n):
                if i != 5:
                    assert torch.equal(pages[slots[i] // 16, :, slots[i] % 16], rows[i]), i
            assert float(pages[3, :, 5].abs().max()) == 0 and float(pages[0].abs().max()) == 0
        assert ops.head_rotary_norm(join([q, k, v]).to(device), H, G, dim, vdim, cos.to(device), sin.to(device), pos.to(device), 1e-3, kp, vp,
                                    slots.to(device), False)[1] is None


def paged(rows, ids, extra=0):
    """Cache pages holding ``rows[n, G, size]`` in the given page order."""
    n, G, size = rows.shape
    pages = torch.zeros(max(ids) + 1 + extra, G, 16, size, dtype=rows.dtype)
    for i in range(n):
        pages[ids[i // 16], :, i % 16] = rows[i]
    return pages


def check_attention(ops, device, dtype, H, G, dim, vdim, chunk, cap, size=0, ctx=300):
    """One key per query stands out.  It is found wherever it lies inside the query's chunk, and from the next chunk or from in front of
    it the result is that of the other keys; queries alone, in portions and packed, through the paged cache and gathered."""
    g = torch.Generator().manual_seed(chunk + dim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    kd, vd = (size, size) if size else (up8(dim), up8(vdim))
    padc = lambda t, n: torch.cat([t, torch.zeros(*t.shape[:-1], n - t.shape[-1], dtype=t.dtype)], -1)
    unit = lambda t: t / t.norm(dim=-1, keepdim=True)
    k, v = unit(rnd(ctx, G, dim)).to(dtype), rnd(ctx, G, vdim).to(dtype)
    ids = torch.randperm((ctx + 15) // 16 + 3, generator=g).tolist()[: (ctx + 15) // 16]
    kp, vp = paged(padc(k, kd), ids, 2).to(device), paged(padc(v, vd), ids, 2).to(device)
    table = torch.tensor([ids], dtype=torch.int32, device=device)
    scale, cols = (2.0 if cap else 1.0), up8(vdim)
    tol = 0.02 if dtype == torch.bfloat16 else 2e-5
    kf, vf = k.double(), v.double()
    c = chunk or 64
    spots = sorted({0, 1, 15, 16, 17, c - 1, c, c + 1, 2 * c - 1, 2 * c, ctx - 2, ctx - 1} & set(range(ctx)))
    for mark in spots:
        lasts = sorted({mark, max(mark - 1, 0), min(mark // c * c + c - 1, ctx - 1), min(mark // c * c + c, ctx - 1), ctx - 1})
        for last in lasts:
            for n in (1, 2, 20):
                if n > last + 1:
                    continue
                q = (k[mark].float() * 25.0).repeat_interleave(H // G, 0).to(dtype).repeat(n, 1, 1)
                gate = rnd(n, H).to(dtype)
                want = oracle.attend(q.double(), kf[: last + 1], vf[: last + 1], scale, cap, chunk, last + 1 - n)
                want = want / (1 + torch.exp(-gate.double()))[..., None]
                cu = torch.tensor([0, n], dtype=torch.int32, device=device)
                out = ops.paged_attention(padc(q, kd).to(device), kp, vp, table, torch.tensor([last + 1], dtype=torch.int32, device=device),
                                          cu if n > 1 else None, ctx, scale, cap, chunk, gate.to(device), vdim, cols)
                out = out.view(n, H, cols).double().cpu()
                assert float((out[..., :vdim] - want).abs().max()) < tol * 3, (mark, last, n)
                assert cols == vdim or float(out[..., vdim:].abs().max()) == 0
                if n == 1 and not cap:
                    seen = mark <= last and (not chunk or mark // chunk == last // chunk)
                    w = torch.softmax((kf[:, 0] @ q[0, 0].double()) * scale, 0)[mark] if seen else 0
                    assert (float(w) > 0.5) == seen          # the marked key does stand out
    if not size:
        return
    # packed: every chunk a sequence of its own, keys gathered from the pages
    chunk = chunk or ctx
    for first, n in ((0, ctx), (c - 1, 2), (c, 30), (c + 5, ctx - c - 5), (ctx - 20, 20)):
        cq, ck, seq, firsts, at = [0], [0], [], [], first
        while at < first + n:
            lo = at // chunk * chunk
            end = min(first + n, lo + chunk)
            cq.append(cq[-1] + end - at)
            ck.append(ck[-1] + end - lo)
            seq.append(0)
            firsts.append(lo)
            at = end
        t = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
        kk, vv = ops.kv_gather(kp, vp, table, t(seq), t(firsts), t(ck), ck[-1])
        pick = torch.cat([torch.arange(f, f + y - x) for f, x, y in zip(firsts, ck, ck[1:])])
        assert torch.equal(kk.cpu(), padc(k, kd)[pick]) and torch.equal(vv.cpu(), padc(v, vd)[pick])
        q, gate = unit(rnd(n, H, dim)).mul(12.0).to(dtype), rnd(n, H + 2).to(dtype)[:, 1:H + 1]
        want = oracle.attend(q.double(), kf[: first + n], vf[: first + n], scale, cap, chunk, first) / (1 + torch.exp(-gate.double()))[..., None]
        for bound in (0.0, 12.5 * scale):
            out = ops.attention_context(padc(q, kd).to(device), kk, vv, t(cq), t(ck), max(y - x for x, y in zip(cq, cq[1:])), scale, cap,
                                        gate.to(device), cols, bound).double().cpu()
            assert float((out[..., :vdim] - want).abs().max()) < tol * 3, (first, n, bound)


def delta_case(H, G, d, dv, taps, lens, seed=0, a_log=None, alike=0.0, dtype=torch.float32):
    """Random inputs of the recurrence for sequences with ``lens`` tokens.  ``alike``: 0 .. 1, how much the keys resemble one another."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    n = sum(lens)
    parts = [rnd(n, G * d), rnd(n, G * d), rnd(n, H * dv), rnd(n, H * dv), rnd(n, H), rnd(n, H)]
    if alike:
        parts[1] = alike * rnd(1, G * d) + (1 - alike) * parts[1]
        parts[4] = parts[4] + 4.0
    w = dict(conv=rnd(taps, 2 * G * d + H * dv) * taps ** -0.5, a_log=torch.full((H,), float(a_log)) if a_log is not None else rnd(H) - 1.0,
             dt=rnd(H), norm=1 + 0.1 * rnd(dv))
    return [p.to(dtype) for p in parts], w


def delta_oracle(parts, w, H, G, d, dv, eps, lo, hi):
    """The plain recurrence on one sequence's rows: the mixer with identity projections."""
    x = [p[lo:hi].double() for p in parts]
    c = w["conv"].double().t()
    q, k, v = (oracle.silu(oracle.short_conv(t, c[a:b])) for t, a, b in ((x[0], 0, G * d), (x[1], G * d, 2 * G * d), (x[2], 2 * G * d, None)))
    n = hi - lo
    q, k, v = oracle.unit(q.view(n, G, d)) / math.sqrt(d), oracle.unit(k.view(n, G, d)), v.view(n, H, dv)
    beta, g = 1 / (1 + torch.exp(-x[4])), oracle.decay(x[5], w["a_log"].double(), w["dt"].double())
    out, states = [], []
    for a in range(H):
        o, S = oracle.delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], g[:, a])
        out.append(oracle.rms(o, w["norm"].double(), eps) * oracle.silu(x[3].view(n, H, dv)[:, a]))
        states.append(S)
    return torch.cat(out, -1), torch.stack(states)


def run_delta(ops, device, parts, w, H, G, d, dv, eps, sequences, cuts, slots):
    """Feeds each sequence in portions (``cuts``: lists of tokens per pass, one entry per sequence) through one state cache; returns
    outputs per sequence and the states."""
    taps = w["conv"].shape[0]
    dt = parts[0].dtype
    ns = max(slots) + 2
    state = torch.full((ns, H, d, (dv + 3) // 4 * 4), 9.0, device=device)
    ring = torch.full((ns, H, max(taps - 1, 1), 2 * d + dv), 9.0, device=device, dtype=dt)
    rows = join(parts)
    at, outs = [0] * len(sequences), [[] for _ in sequences]
    for step in cuts:
        live = [i for i, m in enumerate(step) if m]
        pick = torch.cat([torch.arange(sequences[i][0] + at[i], sequences[i][0] + at[i] + step[i]) for i in live])
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
        cu, ctx = [0], []
        for i in live:
            cu.append(cu[-1] + step[i])
            ctx.append(at[i] + step[i])
        single = all(step[i] == 1 for i in live)
        o = ops.delta_rule(rows[pick].to(device), H, G, d, dv, *(w[x].to(device) for x in ("conv", "a_log", "dt", "norm")), eps, state, ring,
                           i32([slots[i] for i in live]), None if single else i32(cu), i32(ctx), max(step[i] for i in live))
        for j, i in enumerate(live):
            outs[i].append(o[cu[j]:cu[j + 1], : H * dv].double().cpu())
            at[i] += step[i]
    return [torch.cat(o) for o in outs], state.double().cpu()


def check_delta(ops, device, dtype, H, G, d, dv, taps, lens, cuts, a_log=None, alike=0.0):
    parts, w = delta_case(H, G, d, dv, taps, lens, sum(lens), a_log, alike, dtype)
    sequences = [(sum(lens[:i]), sum(lens[:i + 1])) for i in range(len(lens))]
    slots = torch.randperm(len(lens) + 1, generator=torch.Generator().manual_seed(1)).tolist()[: len(lens)]
    outs, state = run_delta(ops, device, parts, w, H, G, d, dv, 1e-4, sequences, cuts, slots)
    for i, (lo, hi) in enumerate(sequences):
        want, S = delta_oracle(parts, w, H, G, d, dv, 1e-4, lo, hi)
        n = outs[i].shape[0]
        assert n == hi - lo
        e = (outs[i] - want).norm(dim=-1) / want.norm(dim=-1)
        es = float((state[slots[i]][..., :dv] - S).norm() / S.norm())
        # the output norm divides by what may be a small read-out: single rows may be further off in bf16
        most, worst, states = (0.02, 0.12, 0.01) if dtype == torch.bfloat16 else (2e-5, 3e-5, 2e-5)
        more = 4 if alike else 1
        assert float(e.quantile(0.9)) < most * more and float(e.max()) < worst * more and es < states * more, (
            i, float(e.quantile(0.9)), float(e.max()), int(e.argmax()), es)


DELTA_CASES = [  # heads, query/key heads, sizes, taps, tokens of the sequences, passes, A_log, likeness of the keys
    (2, 1, 12, 20, 4, [70, 5], [[30, 0], [1, 1], [1, 1], [2, 3], [36, 0]], None, 0.0),
    (2, 2, 64, 64, 4, [130], [[130]], None, 0.0),
    (4, 2, 64, 72, 3, [63, 64, 65, 1], [[63, 64, 65, 1]], None, 0.0),
    (2, 1, 128, 128, 4, [129, 128], [[64, 1], [65, 127]], -7.0, 0.0),          # nearly no decay
    (2, 1, 128, 64, 2, [100, 33], [[100, 33]], 3.0, 0.0),                      # states that die within a token or two
    (1, 1, 40, 136, 1, [90], [[17], [2], [1], [70]], None, 0.0),               # no convolution history
    (2, 2, 128, 128, 4, [150], [[150]], -7.0, 0.95),                           # keys nearly alike, steps near one
    (2, 2, 24, 8, 4, [64, 2], [[2, 2], [62, 0]], None, 0.0),                   # a pass shorter than the convolution
    (1, 1, 264, 260, 5, [8], [[4], [1], [3]], None, 0.0),                      # beyond what the kernels keep on chip
]
ATTENTION_CASES = [  # heads, KV heads, sizes, chunk, cap, size in the tensor-core kernels
    (2, 1, 64, 64, 37, 0.0, 64), (6, 2, 96, 80, 64, 30.0, 128), (5, 5, 40, 24, 1, 2.0, 64), (11, 1, 128, 128, 100, 50.0, 128), (4, 2, 56, 64, 0, 0.0, 64),
    (2, 1, 20, 9, 33, 8.0, 0), (3, 1, 136, 152, 48, 0.0, 0)]

#!/usr/bin/env python3
"""Speed of the Vunitar design beside the framework's closest model (the Llama family without depth routing) at equal
width, heads and active parameters per token; random weights.

    python benchmarks/vunitar_bench.py                  # kernels one by one, then prefill and decode through the engine
    python benchmarks/vunitar_bench.py --only kernels

Kernels: device time from a CUDA graph of many launches over rotating buffers (the working set exceeds the 126 MB L2),
and the fraction of the measured copy bandwidth or matrix throughput (``MEASURED_PEAKS.json``) that the algorithm's
bytes or FLOPs come to.  Engine: wall clock with a device synchronize on both sides.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "benchmarks"))
from compare_common import engine_arm, peaks, timed  # noqa: E402
from kotodama_b200.config import ModelConfig  # noqa: E402
from kotodama_b200.models.llama import KotodamaModel  # noqa: E402
from kotodama_b200.models.vunitar import VunitarConfig, VunitarModel  # noqa: E402

VOCAB = 49152
# name -> width, heads, kv_rank, layers, experts, top, expert ff, shared ff, dense ff (layer 0; all layers when experts = 0), KV heads of the Llama arm
SIZES = {
    "2048-moe": dict(width=2048, heads=16, rank=512, layers=8, experts=64, top=6, ff=1408, shared=2816, dense=11264, kv=4),
    "3072-moe": dict(width=3072, heads=24, rank=512, layers=6, experts=64, top=8, ff=1024, shared=2048, dense=10240, kv=8),
    "4096-dense": dict(width=4096, heads=32, rank=512, layers=6, experts=0, top=0, ff=0, shared=0, dense=16384, kv=8),
}


def vunitar_config(z: dict) -> VunitarConfig:
    mixer = dict(heads=z["heads"], dim=128, vdim=128, kv_rank=z["rank"], scale=128 ** -0.5)
    dense = dict(kind="dense", ff=z["dense"])
    moe = dict(kind="moe", expert=dict(ff=z["ff"]), shared=dict(ff=z["shared"]),
               router=dict(experts=z["experts"], top=z["top"], scale=1.0, groups=dict(count=8, keep=4)))
    layers = [dict(type="latent_attention", mixer=mixer, mlp=dense if i == 0 or not z["experts"] else moe) for i in range(z["layers"])]
    return VunitarConfig.from_dict(dict(architecture="Vunitar", vocab=VOCAB, width=z["width"], norm=dict(eps=1e-5), logit_softcap=30.0,
                                        embedding=dict(bigram=dict(buckets=65521, mul_prev=131, mul_cur=31)), layers=layers))


def llama_config(z: dict) -> ModelConfig:
    """Same width and heads; a SwiGLU of as many active parameters as the expert (or dense) layers of the other arm."""
    active = z["top"] * z["ff"] + z["shared"] if z["experts"] else z["dense"]
    inter = (active * 2 // 3 + 127) // 128 * 128
    return ModelConfig(hidden_size=z["width"], num_layers=z["layers"], num_attention_heads=z["heads"], num_kv_heads=z["kv"],
                       head_dim=128, intermediate_size=inter, vocab_size=VOCAB, max_position_embeddings=8192, tie_word_embeddings=True)


def kernels(name: str, z: dict, batch: int = 64, ctx: int = 1280, tokens: int = 8192) -> list[dict]:
    from kotodama_b200.ops import get_ops
    ops = get_ops("cuda")
    pk = peaks()
    dev = "cuda"
    D, H, R = z["width"], z["heads"], z["rank"]
    bf = lambda *s: torch.randn(*s, device=dev, dtype=torch.bfloat16)
    out = []

    def add(kernel: str, like: str, ms: float, nbytes: float = 0.0, flops: float = 0.0) -> None:
        t_mem, t_mma = nbytes / (pk["gbs"] * 1e9), flops / (pk["tflops"] * 1e12)
        bound = max(t_mem, t_mma)
        out.append(dict(size=name, kernel=kernel, like=like, us=round(ms * 1e3, 2), bound="memory" if t_mem >= t_mma else "matrix",
                        roofline_us=round(bound * 1e6, 2), frac=round(bound / (ms * 1e-3), 3)))

    # ---- decode attention: B sequences of `ctx` cached tokens each
    B, mp = batch, (ctx + 15) // 16
    sets = max(2, int(400e6 // (B * ctx * R * 2)) + 1)
    lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
    tables = torch.randperm(B * mp, device=dev).to(torch.int32).view(B, mp).contiguous()
    pages = [bf(B * mp, R // 64, 16, 64) for _ in range(sets)]
    q = bf(B, H, R)
    ms = timed([lambda i=i: ops.latent_attention(q, pages[i], tables, lens, None, 1, ctx, 0.088) for i in range(sets)])
    add("latent decode attention + merge", "decode attention", ms, B * ctx * R * 2 + 2 * B * H * R * 2, 4.0 * B * ctx * H * R)
    del pages
    KV = z["kv"]
    sets = max(2, int(400e6 // (B * ctx * KV * 128 * 4)) + 1)
    kp = [(bf(B * mp, KV, 16, 128), bf(B * mp, KV, 16, 128)) for _ in range(sets)]
    ql = bf(B, H * 128)
    ms = timed([lambda i=i: ops.paged_decode_attention(ql, kp[i][0], kp[i][1], tables, lens, ctx, H, KV, 128) for i in range(sets)])
    add("llama: GQA decode attention + merge", "decode attention", ms, B * ctx * KV * 128 * 4 + 2 * B * H * 128 * 2, 4.0 * B * ctx * H * 128)
    del kp
    # ---- absorbing products of decoding (one small product per head)
    wk = [bf(H, 128, R) for _ in range(max(2, int(300e6 // (H * 128 * R * 2))))]
    qh = bf(B, H, 128)
    oc = bf(B, H, R)
    ms = timed([lambda w=w: ops.head_gemm(qh, w, transposed=True) for w in wk])
    add("per-head product q W_uk (decode)", "decode product", ms, H * 128 * R * 2 + B * H * (128 + R) * 2, 2.0 * B * H * 128 * R)
    ms = timed([lambda w=w: ops.head_gemm(oc, w) for w in wk])
    add("per-head product W_uv o (decode)", "decode product", ms, H * 128 * R * 2 + B * H * (128 + R) * 2, 2.0 * B * H * 128 * R)
    del wk
    # ---- decode products: a dense projection of the Llama arm and the experts
    cfg = llama_config(z)
    F = cfg.intermediate_size
    ws = [ops.decode_weight(bf(2 * F, D)) for _ in range(max(2, int(400e6 // (2 * F * D * 2)) + 1))]
    a = bf(B, D)
    ms = timed([lambda w=w: ops.gemm_nt(a, w) for w in ws])
    add("llama: gate|up projection (decode)", "decode product", ms, 2 * F * D * 2 + B * (D + 2 * F) * 2, 4.0 * B * F * D)
    nq = H * 128 + R
    ws = [ops.decode_weight(bf(nq, D)) for _ in range(max(2, int(400e6 // (nq * D * 2)) + 1))]
    ms = timed([lambda w=w: ops.gemm_nt(a, w) for w in ws])
    add("q | latent projection (decode)", "decode product", ms, nq * D * 2 + B * (D + nq) * 2, 2.0 * B * nq * D)
    nq = (H + 2 * KV) * 128
    ws = [ops.decode_weight(bf(nq, D)) for _ in range(max(2, int(400e6 // (nq * D * 2)) + 1))]
    ms = timed([lambda w=w: ops.gemm_nt(a, w) for w in ws])
    add("llama: q | k | v projection (decode)", "decode product", ms, nq * D * 2 + B * (D + nq) * 2, 2.0 * B * nq * D)
    # what small decode launches cost in the Llama family: a product of about the bytes of a per-head product, row kernels
    ws = [ops.decode_weight(bf(512, D)) for _ in range(64)]
    ms = timed([lambda w=w: ops.gemm_nt(a, w) for w in ws])
    add("llama: k or v projection alone (decode)", "decode product", ms, 512 * D * 2 + B * (D + 512) * 2, 2.0 * B * 512 * D)
    del ws
    xs, one = [bf(B, D) for _ in range(8)], torch.ones(D, device=dev, dtype=torch.bfloat16)
    ms = timed([lambda x=x: ops.route_norm_fwd([x], None, None, one, 1e-5) for x in xs])
    add("llama: RMS norm (decode)", "row kernel", ms, B * D * 4)
    gus = [bf(B, 2 * F) for _ in range(8)]
    ms = timed([lambda x=x: ops.swiglu_fwd(x) for x in gus])
    add("llama: SwiGLU (decode)", "row kernel", ms, B * 3 * F * 2)
    xf, ones = [torch.randn(B, D, device=dev) for _ in range(8)], torch.ones(D, device=dev)
    ms = timed([lambda x=x: ops.norm_add(x, a, ones, D, 1e-5) for x in xf])
    add("norm + layer scale + residual (decode)", "row kernel", ms, B * D * 12)
    if z["experts"]:
        E, top, ff = z["experts"], z["top"], z["ff"]
        for n, tag, like in ((B, "decode", "decode product"), (tokens, "prefill", "product")):
            A = n * top
            sets = max(2, int(600e6 // (E * ff * D * 2)) + 1) if n == B else 2
            up = [bf(E, ff, D) for _ in range(sets)]
            ids = torch.stack([torch.randperm(E, device=dev)[:top] for _ in range(n)]).to(torch.int32)
            h = bf(n, D)
            _, at = ops.moe_experts(h, ids, up[0], up[0].view(E, D, ff), "gelu")
            cnt = torch.bincount(ids.flatten().long(), minlength=E)
            off = torch.cat([torch.zeros(1, device=dev, dtype=torch.long), cnt.cumsum(0)]).to(torch.int32)
            rows, u = bf(A, D), bf(A, ff)
            live = int((cnt > 0).sum())
            ms = timed([lambda w=w: ops._grouped(rows, w, off, "gelu") for w in up])
            add(f"expert up + GELU ({tag})", like, ms, (live * ff * D + A * (D + ff)) * 2, 2.0 * A * D * ff)
            ms = timed([lambda w=w: ops._grouped(u, w.view(E, D, ff), off, None) for w in up])
            add(f"expert down ({tag})", like, ms, (live * ff * D + A * (D + ff)) * 2, 2.0 * A * D * ff)
            router = bf(E + 1, D)
            hs = [bf(n, D) for _ in range(4)]
            ms = timed([lambda x=x: ops.moe_route(x, router, E, top, 1.0, 8, 4) for x in hs])
            add(f"router + selection ({tag})", "row kernel", ms, (n * D + (E + 1) * D) * 2, 2.0 * n * D * (E + 1))
            plans = [ops.moe_route(x, router, E, top, 1.0, 8, 4) for x in hs]
            # grouping turns the plan's ranks into places: every replay starts from a copy of the ranks
            keep = [(p[3][0], p[3][1].clone()) if p[3] is not None else None for p in plans]
            group = lambda x, p, k: ops._moe_group(x, p[0], E, None if k is None else (k[0], k[1].clone()))
            ms = timed([lambda x=x, p=p, k=k: group(x, p, k) for x, p, k in zip(hs, plans, keep)])
            add(f"grouping + row gather ({tag})", "row kernel", ms, (n * D + A * D) * 2)
            xs = [torch.randn(n, D, device=dev) for _ in range(4)]
            ye, ys, wts, gate, g = bf(A, D), bf(n, D), torch.rand(n, top, device=dev), torch.rand(n, device=dev), torch.ones(D, device=dev)
            ms = timed([lambda x=x: ops.moe_combine_norm_add(x, ye, at, wts, ys, gate, g, D, 1e-5, torch.bfloat16) for x in xs])
            add(f"combine + norm + residual ({tag})", "row kernel", ms, A * D * 2 + n * D * (2 + 4 + 4 + 2))
            del up, rows, u, ye
    # ---- prefill: attention, dense product, row kernels
    n = tokens
    qf, kf, vf = bf(n, H, 128), bf(n, H, 128), bf(n, H, 128)
    cu = torch.tensor([0, n // 2, n], dtype=torch.int32, device=dev)
    T = n // 2
    fl = 2 * 4.0 * H * 128 * T * (T + 1) / 2
    ms = timed([lambda: ops.attention_context(qf, kf, vf, cu, cu, T, 0.088) for _ in range(2)])
    add("flash attention, expanded latents (prefill)", "attention", ms, n * H * 128 * 8, fl)
    ql, kl, vl = bf(1, n, H, 128), bf(1, n, KV, 128), bf(1, n, KV, 128)
    ms = timed([lambda: ops.attention_fwd(ql, kl, vl, need_grad=False, cu_seqlens=cu, max_seqlen=T) for _ in range(2)])
    add("llama: flash attention (prefill)", "attention", ms, n * (2 * H + 2 * KV) * 256, fl)
    c, wkv = bf(n, R), bf(2 * H * 128, R)
    ms = timed([lambda: ops.gemm_nt(c, wkv) for _ in range(3)])
    add("latent expansion c -> k | v (prefill)", "product", ms, (n * R + 2 * H * 128 * (n + R)) * 2, 2.0 * n * R * 2 * H * 128)
    a, w = bf(n, D), bf(2 * F, D)
    ms = timed([lambda: ops.gemm_nt(a, w) for _ in range(2)])
    add("llama: gate|up projection (prefill)", "product", ms, (n * D + 2 * F * (n + D)) * 2, 4.0 * n * D * F)
    gu = bf(n, 2 * F)
    ms = timed([lambda: ops.swiglu_fwd(gu) for _ in range(2)])
    add("llama: SwiGLU (prefill)", "row kernel", ms, n * 3 * F * 2)
    ud = bf(n, z["dense"])
    ms = timed([lambda: ops.activate(ud, "relu2") for _ in range(2)])
    add("squared ReLU (prefill)", "row kernel", ms, n * z["dense"] * 4)
    if z["shared"]:
        us = bf(n, z["shared"])
        ms = timed([lambda: ops.activate(us, "gelu") for _ in range(6)])
        add("GELU (prefill)", "row kernel", ms, n * z["shared"] * 4)
    xs, y, g = [torch.randn(n, D, device=dev) for _ in range(3)], bf(n, D), torch.ones(D, device=dev)
    ms = timed([lambda x=x: ops.norm_add(x, y, g, D, 1e-5) for x in xs])
    add("norm + layer scale + residual (prefill)", "row kernel", ms, n * D * (2 + 4 + 4 + 2))
    xb, nw = [bf(n, D) for _ in range(4)], torch.ones(D, device=dev, dtype=torch.bfloat16)
    ms = timed([lambda x=x: ops.route_norm_fwd([x], None, None, nw, 1e-5) for x in xb])
    add("llama: RMS norm (prefill)", "row kernel", ms, n * D * 4)
    qc = [bf(n, H * 128 + R) for _ in range(3)]
    pg = torch.zeros(n // 16, R // 64, 16, 64, device=dev, dtype=torch.bfloat16)
    sl, cw = torch.arange(n, device=dev), torch.ones(R, device=dev)
    ms = timed([lambda x=x: ops.latent_append(x[:, H * 128:], cw, R, 1e-5, pg, sl) for x in qc])
    add("latent norm + cache append (prefill)", "row kernel", ms, n * R * 6)
    ops.check_status()
    return out


def engines(name: str, z: dict, requests: int = 64, prompt: int = 1024, new: int = 48) -> dict:
    vc, lc = vunitar_config(z), llama_config(z)
    out = dict(size=name, requests=requests, prompt_tokens=prompt, new_tokens=new, vunitar_params=vc.param_count(),
               llama_params=lc.param_count())
    out["vunitar"] = engine_arm(VunitarModel.random_init(vc, 0, device="cuda"), requests, prompt, new)
    torch.cuda.empty_cache()
    with torch.device("meta"):
        m = KotodamaModel(lc)
    out["llama"] = engine_arm(m, requests, prompt, new)
    return out


def run(sizes: list[str], only: str = "") -> dict:
    res = dict(kernels=[], engines=[], peaks=peaks())
    for name in sizes:
        if only in ("", "kernels"):
            res["kernels"] += kernels(name, SIZES[name])
            torch.cuda.empty_cache()
        if only in ("", "engines"):
            res["engines"].append(engines(name, SIZES[name]))
    return res


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default=",".join(SIZES))
    ap.add_argument("--only", default="", choices=["", "kernels", "engines"])
    a = ap.parse_args()
    res = run(a.sizes.split(","), a.only)
    for k in res["kernels"]:
        print(f"{k['size']:<12}{k['kernel']:<46}{k['like']:<18}{k['us']:>9.1f} us  roofline {k['roofline_us']:>9.1f} us ({k['bound']})  {k['frac']:.3f}")
    for e in res["engines"]:
        print(json.dumps(e))


if __name__ == "__main__":
    main()

#!/usr/bin/env python3
"""Speed of the Lisunex design beside the framework's closest model (the Llama family without depth routing) at equal
width, heads, feed-forward and number of layer runs; random weights.

    python benchmarks/lisunex_bench.py                  # kernels one by one, then prefill and decode through the engine
    python benchmarks/lisunex_bench.py --only kernels

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
from compare_common import engine_arm, kernel_ms, peaks, timed  # noqa: E402
from kotodama_b200.config import ModelConfig  # noqa: E402
from kotodama_b200.models.lisunex import LisunexConfig, LisunexModel  # noqa: E402
from kotodama_b200.models.llama import KotodamaModel  # noqa: E402

VOCAB = 49152
# width, attention heads and KV heads, delta heads and their query/key heads, feed-forward, layers in front of / in / behind the loop (each a
# delta layer and an attention layer, the looped ones run twice)
SIZES = {
    "2048": dict(width=2048, heads=16, kv=4, dheads=16, dkv=16, ff=8192, blocks=(1, 1, 1)),
    "3072": dict(width=3072, heads=24, kv=8, dheads=24, dkv=12, ff=8192, blocks=(1, 1, 0)),
    "4096": dict(width=4096, heads=32, kv=8, dheads=32, dkv=16, ff=14336, blocks=(1, 1, 0)),
}
CHUNK, TAPS, CAP = 2048, 4, 30.0


def lisunex_config(z: dict) -> LisunexConfig:
    delta = dict(type="delta", mixer=dict(heads=z["dheads"], kv_heads=z["dkv"], dim=128, vdim=128, conv=TAPS))
    attn = dict(type="attention", mixer=dict(heads=z["heads"], kv_heads=z["kv"], dim=128, vdim=128, scale=128 ** -0.5, softcap=CAP,
                                             mask=dict(size=CHUNK), rot=dict(dims=128, base=10000.0, scaling=dict(
                                                 factor=4.0, original=2048, fast=32.0, slow=1.0))))
    layers = [dict(m, mlp=dict(kind="dense", ff=z["ff"])) for _ in range(sum(z["blocks"])) for m in (delta, attn)]
    a, b, _ = z["blocks"]
    return LisunexConfig.from_dict(dict(architecture="Lisunex", vocab=VOCAB, width=z["width"], norm=dict(eps=1e-5), embedding=dict(scale=1.0),
                                        layers=layers, loop=dict(start=2 * a, stop=2 * (a + b), times=2)))


def llama_config(z: dict) -> ModelConfig:
    runs = 2 * (sum(z["blocks"]) + z["blocks"][1])
    return ModelConfig(hidden_size=z["width"], num_layers=runs, num_attention_heads=z["heads"], num_kv_heads=z["kv"], head_dim=128,
                       intermediate_size=z["ff"], vocab_size=VOCAB, max_position_embeddings=8192, tie_word_embeddings=True)


def kernels(name: str, z: dict, batch: int = 64, ctx: int = 1280, tokens: int = 8192) -> list[dict]:
    from kotodama_b200.ops import get_ops
    ops = get_ops("cuda")
    pk = peaks()
    dev = "cuda"
    D, H, KV, DH, DG, F = z["width"], z["heads"], z["kv"], z["dheads"], z["dkv"], z["ff"]
    bf = lambda *s: torch.randn(*s, device=dev, dtype=torch.bfloat16)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    out = []

    def add(kernel: str, like: str, ms: float, nbytes: float = 0.0, flops: float = 0.0) -> None:
        t_mem, t_mma = nbytes / (pk["gbs"] * 1e9), flops / (pk["tflops"] * 1e12)
        bound = max(t_mem, t_mma)
        out.append(dict(size=name, kernel=kernel, like=like, us=round(ms * 1e3, 2), bound="memory" if t_mem >= t_mma else "matrix",
                        roofline_us=round(bound * 1e6, 2), frac=round(bound / (ms * 1e-3), 3)))

    # ---- decode attention: B sequences, `ctx` visible keys each
    B, mp = batch, (ctx + 15) // 16
    sets = max(2, int(400e6 // (B * ctx * KV * 128 * 4)) + 1)
    kp = [(bf(B * mp, KV, 16, 128), bf(B * mp, KV, 16, 128)) for _ in range(sets)]
    lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
    tables = torch.randperm(B * mp, device=dev).to(torch.int32).view(B, mp).contiguous()
    q3, ql, gate = bf(B, H, 128), bf(B, H * 128), bf(B, H)
    nbytes = B * ctx * KV * 128 * 4 + 2 * B * H * 128 * 2
    ms = timed([lambda i=i: ops.paged_attention(q3, kp[i][0], kp[i][1], tables, lens, None, ctx, 0.088, CAP, CHUNK, gate, 128, 128)
                for i in range(sets)])
    add("chunked, capped, gated decode attention + merge", "decode attention", ms, nbytes, 4.0 * B * ctx * H * 128)
    ms = timed([lambda i=i: ops.paged_decode_attention(ql, kp[i][0], kp[i][1], tables, lens, ctx, H, KV, 128) for i in range(sets)])
    add("llama: GQA decode attention + merge", "decode attention", ms, nbytes, 4.0 * B * ctx * H * 128)
    del kp
    # ---- the recurrence: one token of B sequences, then whole prompts
    W = 2 * DG * 128 + 2 * DH * 128 + 2 * DH
    conv = torch.randn(TAPS, (2 * DG + DH) * 128, device=dev) * 0.5
    al, dt, nw = torch.randn(DH, device=dev) - 1, torch.randn(DH, device=dev), torch.ones(128, device=dev)
    rows = [bf(B, W) for _ in range(4)]
    slots = torch.arange(B, dtype=torch.int32, device=dev)
    sets = 4
    st = [torch.randn(B, DH, 128, 128, device=dev) * 0.1 for _ in range(sets)]
    rg = [bf(B, DH, TAPS - 1, 384) for _ in range(sets)]
    ms = timed([lambda i=i: ops.delta_rule(rows[i], DH, DG, 128, 128, conv, al, dt, nw, 1e-5, st[i], rg[i], slots, None, lens, 1) for i in range(sets)])
    add("delta rule, one token", "decode attention", ms, B * (DH * 128 * 128 * 8 + DH * 384 * (2 * TAPS - 2) * 2 + W * 2 + DH * 256))
    n = tokens
    cu, ctxs = i32([0] + [(i + 1) * 1024 for i in range(n // 1024)]), i32([1024] * (n // 1024))
    rows = [bf(n, W) for _ in range(3)]
    # products of the chunked form, every operand counted once
    fl = n * DH * (2.0 * 128 * 64 * 128 + 2.0 * 128 * 128 * 128 + 2.0 * 128 * 64 * 128 * 2 + 2.0 * 64 ** 3) / 64
    calls = [lambda r=r: ops.delta_rule(r, DH, DG, 128, 128, conv, al, dt, nw, 1e-5, st[0], rg[0], slots[: n // 1024], cu, ctxs, 1024) for r in rows]
    add("delta rule, prompts of 1024 (all launches)", "attention", timed(calls), n * (W + DH * 128) * 2 + n // 1024 * DH * 128 * 128 * 4, fl)
    # its launches one by one, each against the bytes and products of its own inputs and outputs
    part = kernel_ms(calls * 3, ["delta_conv", "delta_prepare", "delta_scan", "delta_finish"])
    qk, vo, tt = n * 2 * DG * 256, n * DH * 256, n // 64 * DH * 32768
    add("  delta conv + SiLU", "row kernel", part["delta_conv"], 2 * (qk + vo))
    add("  delta prepare (triangular inverses)", "attention", part["delta_prepare"], qk + tt, n // 64 * DH * (2.0 * 128 * 64 * 128 + 2.0 * 64 ** 3))
    add("  delta scan", "attention", part["delta_scan"], qk + 2 * vo + tt, n // 64 * DH * (2.0 * 128 * 128 * 128 + 2 * 2.0 * 128 * 64 * 128))
    add("  delta output norm + gate", "row kernel", part["delta_finish"], 3 * vo)
    del st, rg
    # ---- decode products and row kernels
    a = bf(B, D)
    for tag, N in (("q | k | v | g of attention", (H + 2 * KV) * 128 + H), ("q | k | v | g | b | a of delta", W), ("llama: q | k | v", (H + 2 * KV) * 128),
                   ("gate|up", 2 * F)):
        ws = [ops.decode_weight(bf(N, D)) for _ in range(max(2, int(400e6 // (N * D * 2)) + 1))]
        bias = bf(N).expand(B, -1) if "attention" in tag else None
        ms = timed([lambda w=w: ops.gemm_nt(a, w, residual=bias) for w in ws])
        add(f"{tag} projection (decode)", "decode product", ms, N * D * 2 + B * (D + N) * 2, 2.0 * B * N * D)
        del ws
    cos, sin = torch.ones(4096, 64, device=dev), torch.zeros(4096, 64, device=dev)
    cosl, sinl = torch.ones(4096, 128, device=dev), torch.zeros(4096, 128, device=dev)
    for m, tag in ((B, "decode"), (n, "prefill")):
        k = 8 if m == B else 3
        xs, ys, ones = [torch.randn(m, D, device=dev) for _ in range(k)], [bf(m, D) for _ in range(k)], torch.ones(D, device=dev)
        ms = timed([lambda x=x, y=y: ops.add_norm(x, y, None, ones, D, 1e-5, torch.bfloat16) for x, y in zip(xs, ys)])
        add(f"residual + RMS norm ({tag})", "row kernel", ms, m * D * (4 + 4 + 2 + 2))
        oneb = torch.ones(D, device=dev, dtype=torch.bfloat16)
        ms = timed([lambda y=y: ops.route_norm_fwd([y], None, None, oneb, 1e-5) for y in ys])
        add(f"llama: RMS norm ({tag})", "row kernel", ms, m * D * 4)
        del xs, ys
        wq = (H + 2 * KV) * 128
        rows = [bf(m, wq + H) for _ in range(k)]
        pages = [(torch.zeros(m // 16 + 1, KV, 16, 128, device=dev, dtype=torch.bfloat16), torch.zeros(m // 16 + 1, KV, 16, 128, device=dev, dtype=torch.bfloat16))
                 for _ in range(k)]
        pos, sl = torch.arange(m, device=dev, dtype=torch.int32) % 4096, torch.arange(m, device=dev)
        keep = m == n
        ms = timed([lambda i=i: ops.head_rotary_norm(rows[i], H, KV, 128, 128, cos, sin, pos, 1e-5, *pages[i], sl, keep) for i in range(k)])
        add(f"rotary + unit RMS + cache append ({tag})", "row kernel", ms, m * wq * 2 + m * (H + 2 * KV * (2 if keep else 1)) * 256)
        rl, nw2 = [bf(m, wq) for _ in range(k)], torch.ones(128, device=dev, dtype=torch.bfloat16)
        ms = timed([lambda i=i: ops.qknorm_rope_fwd(rl[i], nw2, nw2, cosl, sinl, m, H, KV, 128, 1e-5, positions=pos, append=(*pages[i], sl))
                    for i in range(k)])
        add(f"llama: QK-norm + RoPE + cache append ({tag})", "row kernel", ms, m * wq * 2 + m * (H + KV * 3) * 256)
        del rows, rl, pages
    # ---- prefill attention: two prompts of n / 2, all inside one chunk of the sequence, and chunks of 1024
    qf, kf, vf, gf = bf(n, H, 128), bf(n, KV, 128), bf(n, KV, 128), bf(n, H)
    for T in (n // 2, 1024):
        cu = i32([i * T for i in range(n // T + 1)])
        fl = (n // T) * 4.0 * H * 128 * T * (T + 1) / 2
        for tag, cap, bound in (("capped, gated", CAP, 0.385 * CAP), ("capped (wide scores), gated", CAP, 0.0)):
            ms = timed([lambda: ops.attention_context(qf, kf, vf, cu, cu, T, 0.088, cap, gf, 128, bound) for _ in range(2)])
            add(f"flash attention, {tag}, {T} keys (prefill)", "attention", ms, n * (2 * H + 2 * KV) * 256, fl)
        ms = timed([lambda: ops.attention_fwd(qf[None], kf[None], vf[None], need_grad=False, cu_seqlens=cu, max_seqlen=T) for _ in range(2)])
        add(f"llama: flash attention, {T} keys (prefill)", "attention", ms, n * (2 * H + 2 * KV) * 256, fl)
    # ---- prefill products: with and without the bias in the epilogue
    a = bf(n, D)
    for tag, N, biased in (("q | k | v | g of attention", (H + 2 * KV) * 128 + H, True), ("q | k | v | g | b | a of delta", W, False), ("llama: q | k | v", (H + 2 * KV) * 128, False)):
        w, bias = bf(N, D), bf(N).expand(n, -1) if biased else None
        ms = timed([lambda: ops.gemm_nt(a, w, residual=bias) for _ in range(2)])
        add(f"{tag} projection (prefill)", "product", ms, (n * D + N * (n + D)) * 2, 2.0 * n * D * N)
    ops.check_status()
    return out


def engines(name: str, z: dict, requests: int = 64, prompt: int = 1024, new: int = 48) -> dict:
    xc, lc = lisunex_config(z), llama_config(z)
    out = dict(size=name, requests=requests, prompt_tokens=prompt, new_tokens=new, lisunex_params=xc.param_count(),
               llama_params=lc.param_count(), layer_runs=len(xc.runs()))
    out["lisunex"] = engine_arm(LisunexModel.random_init(xc, 0, device="cuda"), requests, prompt, new)
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
            torch.cuda.empty_cache()
    return res


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default=",".join(SIZES))
    ap.add_argument("--only", default="", choices=["", "kernels", "engines"])
    a = ap.parse_args()
    res = run(a.sizes.split(","), a.only)
    for k in res["kernels"]:
        print(f"{k['size']:<8}{k['kernel']:<64}{k['like']:<18}{k['us']:>9.1f} us  roofline {k['roofline_us']:>9.1f} us ({k['bound']})  {k['frac']:.3f}")
    for e in res["engines"]:
        print(json.dumps(e))


if __name__ == "__main__":
    main()

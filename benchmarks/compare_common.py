"""What the comparisons of a model design with the Llama family share: peaks, kernel timing, the engine arm."""
from __future__ import annotations

import json
import os
import statistics
import sys
import time

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
from kotodama_b200.models.llama import KotodamaModel  # noqa: E402
from kotodama_b200.serve.engine import SamplingParams, ServingEngine  # noqa: E402


def peaks() -> dict:
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as fh:
            d = json.load(fh)
        return {"gbs": d["hbm_gbs"], "tflops": d["bf16_tflops"], "of": "measured"}
    except OSError:
        return {"gbs": 6650.0, "tflops": 1590.0, "of": "fallback"}


def timed(calls: list, reps: int = 5) -> float:
    """Mean device time of one call in ms: the calls (over different buffers) captured in one graph, replayed.  The
    decode kernels of both models are launched as in serving, as programmatic dependents of one another."""
    for c in calls[:2]:
        c()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    from kotodama_b200.ops import get_ops
    with torch.cuda.graph(g), get_ops("cuda").dependent_launch(True):
        keep = [c() for c in calls]
    for _ in range(2):
        g.replay()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(reps):
        g.replay()
    e1.record()
    torch.cuda.synchronize()
    del keep
    return e0.elapsed_time(e1) / (reps * len(calls))


def kernel_ms(calls: list, names: list[str]) -> dict[str, float]:
    """Mean device time in ms of the kernels whose name contains each of ``names``, over the calls (profiler records; for
    operations of several launches)."""
    from torch.profiler import ProfilerActivity, profile
    for c in calls:
        c()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for c in calls:
            c()
        torch.cuda.synchronize()
    out = {}
    for n in names:
        rows = [e for e in prof.key_averages() if n in e.key]
        out[n] = sum(e.self_device_time_total for e in rows) / max(1, sum(e.count for e in rows)) * 1e-3
    return out


def engine_arm(model, requests: int, prompt: int, new: int) -> dict:
    """Prefill of `requests` prompts of `prompt` tokens each, then `new` greedy tokens for all of them."""
    cfg = model.config
    eng = ServingEngine(model, device="cuda", dtype=torch.bfloat16, max_batch=requests, max_ctx=prompt + new + 16)
    if isinstance(model, KotodamaModel):
        eng.arena.init_weights(cfg.num_layers, 0)
    gen = torch.Generator().manual_seed(0)
    prompts = [torch.randint(0, cfg.vocab_size, (prompt,), generator=gen).tolist() for _ in range(requests)]
    res = {}
    for _ in range(2):                                  # the second pass is reported
        before = eng.stats["prefill_s"]
        for p in prompts:
            eng.add_request(p, SamplingParams(max_new_tokens=new, temperature=0.0))
        torch.cuda.synchronize()
        eng.step()
        torch.cuda.synchronize()
        prefill_s = eng.stats["prefill_s"] - before
        eng.graph_ms = []
        steps = []
        while eng.has_work():
            torch.cuda.synchronize()
            t = time.perf_counter()
            eng.step()
            torch.cuda.synchronize()
            steps.append(time.perf_counter() - t)
        res = dict(prefill_tok_s=round(requests * prompt / prefill_s), decode_tok_s=round(requests / statistics.median(steps)),
                   decode_step_ms=round(1e3 * statistics.median(steps), 3), decode_graph_ms=round(statistics.median(eng.graph_ms), 3))
        eng.graph_ms = None
    eng.ops.check_status()
    res["launches"] = eng.ops.launches
    del eng
    torch.cuda.empty_cache()
    return res

"""The Vunitar design on the CPU back end: mechanisms, cache, scheduler, loading, entry points."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import vunitar_cases as cases
from kotodama_b200.ckpt.safetensors import load_safetensors, save_safetensors
from kotodama_b200.models.registry import FAMILIES, load_model, read_config
from kotodama_b200.models.vunitar import VunitarConfig, VunitarModel
from kotodama_b200.ops import get_ops
from kotodama_b200.serve.engine import SamplingParams, ServingEngine

ROOT = Path(__file__).resolve().parents[1]
F32 = torch.float32


def test_row_operations():
    cases.check_ops(get_ops("cpu"), "cpu", F32)


def test_routing_and_experts():
    cases.check_experts(get_ops("cpu"), "cpu", F32)


def test_far_keys_and_the_causal_edge():
    cases.check_far_keys(get_ops("cpu"), "cpu", F32)


@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_prompts_portions_and_decoding(name):
    cases.check_portions(name, "cpu", F32, lengths=(1, 2, 50, 140))


def test_batches_and_reused_pages():
    cases.check_batches("odd", "cpu", F32)


def test_greedy_generation_through_the_scheduler():
    cases.check_generation("odd", "cpu", F32)
    cases.check_generation("plain", "cpu", F32)


def test_portions_interleave_with_decoding_and_cancel_frees_pages():
    cfg = cases.CONFIGS["odd"]
    model = cases.weights(cfg)
    eng = cases.engine(model, "cpu", F32, max_ctx=96, prefill_portion=8)
    short = eng.add_request(cases.tokens(cfg, 4, 0), SamplingParams(max_new_tokens=12, temperature=0.0))
    long = eng.add_request(cases.tokens(cfg, 40, 1), SamplingParams(max_new_tokens=4, temperature=0.0))
    eng.step()
    assert len(short.generated) == 2 and long.ctx_len == 8 and not long.generated
    eng.step()
    assert len(short.generated) == 3 and long.ctx_len == 16        # the short one decodes while the long one is prefilled
    gone = eng.add_request(cases.tokens(cfg, 30, 2), SamplingParams(max_new_tokens=4, temperature=0.0))
    eng.step()
    assert eng.cancel(gone.rid)                                    # in the middle of its prompt
    while eng.has_work():
        eng.step()
    assert short.generated == cases.greedy(cfg, model, short.prompt, 12)
    assert long.generated == cases.greedy(cfg, model, long.prompt, 4)
    assert len(eng.cache.free) == eng.cache.num_pages


def test_sampled_generation_is_reproducible():
    cfg = cases.CONFIGS["plain"]
    eng = cases.engine(cases.weights(cfg), "cpu", F32, max_ctx=96)
    p = SamplingParams(max_new_tokens=10, temperature=0.8, top_k=20, top_p=0.9, repetition_penalty=1.2, seed=5)
    prompt = cases.tokens(cfg, 20, 0)
    a = eng.generate([prompt, prompt], p)
    assert a[0] == a[1] == eng.generate([prompt], p)[0] and len(set(a[0])) > 3


def test_feed_refuses_what_does_not_fit():
    cfg = cases.CONFIGS["odd"]
    eng = cases.engine(cases.weights(cfg), "cpu", F32, max_ctx=32, num_pages=2)
    s = eng.open()
    for toks, places in (([], []), ([cfg["vocab"]], []), ([1, 2], [2]), ([1] * 33, [])):
        with pytest.raises(ValueError):
            eng.feed([(s, toks, places)])
    eng.feed([(s, [1] * 32, [])])
    with pytest.raises(RuntimeError):
        eng.feed([(eng.open(), [1], [])])                          # no page left
    eng.close(s)
    assert len(eng.cache.free) == 2


def test_a_model_that_does_not_continue_a_cache_says_so():
    from kotodama_b200.config import MODEL_PRESETS, ModelConfig
    from kotodama_b200.models.llama import KotodamaModel
    m = lambda: KotodamaModel(ModelConfig(**MODEL_PRESETS["smoke"]))
    with pytest.raises(ValueError):
        ServingEngine(m(), max_batch=1, max_ctx=32, prefill_portion=8)
    with pytest.raises(ValueError):
        ServingEngine(m(), max_batch=1, max_ctx=32).open()


def write_model(folder, cfg, tensors):
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors(tensors, folder / "model.safetensors")
    return folder


def test_model_folders_load_by_architecture(tmp_path):
    cfg = cases.CONFIGS["odd"]
    model = cases.weights(cfg)
    folder = write_model(tmp_path / "v", cfg, model.weights)
    back = load_model(folder)
    assert isinstance(back, VunitarModel) and all(torch.equal(back.weights[k], v) for k, v in model.weights.items())
    assert back.config.param_count() == sum(v.numel() for v in model.weights.values())
    # the Llama family through the same door
    from kotodama_b200.config import MODEL_PRESETS, ModelConfig
    from kotodama_b200.models.llama import KotodamaModel
    lc = ModelConfig(**MODEL_PRESETS["smoke"])
    lm = KotodamaModel(lc)
    state = {k: v for k, v in lm.state_dict().items()}
    lf = write_model(tmp_path / "l", {"architecture": "Kotodama", **lc.to_dict()}, {k: v.clone() for k, v in state.items()})
    assert torch.equal(load_model(lf).embed_tokens.weight, lm.embed_tokens.weight)
    with pytest.raises(ValueError):
        read_config(write_model(tmp_path / "x", {"architecture": "other"}, {"a": torch.zeros(1)}))
    assert {"Kotodama", "Vunitar"} <= set(FAMILIES)


def test_wrong_weights_and_configurations_are_refused(tmp_path):
    cfg = cases.CONFIGS["odd"]
    w = dict(cases.weights(cfg).weights)
    vc = VunitarConfig.from_dict(cfg)
    with pytest.raises(KeyError):
        VunitarModel(vc, {k: v for k, v in w.items() if k != "l0.mix.uk"})
    with pytest.raises(ValueError):
        VunitarModel(vc, {**w, "head": w["head"][:-1]})
    for change in (dict(type="other"), dict(mlp=dict(kind="other")), dict(mlp=cases.moe(6, 5, 8, groups=(3, 2)))):
        with pytest.raises(ValueError):
            VunitarConfig.from_dict({**cfg, "layers": [{**cfg["layers"][0], **change}]})


def test_safetensors_round_trip_and_damage(tmp_path):
    t = {"a": torch.arange(7, dtype=torch.int32), "b": torch.randn(3, 5).bfloat16(), "c": torch.randn(2, 2), "d": torch.zeros(3, dtype=torch.uint8),
         "e": torch.randn(4, dtype=torch.float64)}
    save_safetensors(t, tmp_path / "x.safetensors")
    back = load_safetensors(tmp_path / "x.safetensors")
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) and back[k].dtype == t[k].dtype for k in t)
    raw = (tmp_path / "x.safetensors").read_bytes()
    (tmp_path / "y.safetensors").write_bytes(raw[:-8])
    with pytest.raises(ValueError):
        load_safetensors(tmp_path / "y.safetensors")


def test_trace_replay_program(tmp_path):
    cfg = cases.CONFIGS["plain"]
    model = cases.weights(cfg)
    folder = write_model(tmp_path / "m", cfg, model.weights)
    a, b = cases.tokens(cfg, 20, 0), cases.tokens(cfg, 9, 1)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:12], want=[0, 11])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[12:19], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[19:], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=b, want=[8, 3])], end=["b"])]
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "40", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = cases.oracle_logits(cfg, model, a), cases.oracle_logits(cfg, model, b)
    for step, want, rows in ((0, wa, [0, 11]), (2, wa, [19]), (3, wb, [8, 3])):
        got = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        cases.assert_close(got, want, F32, step, rows)
    assert not (tmp_path / "1.f32").exists()

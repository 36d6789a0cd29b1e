"""The Lisunex design on the CPU back end: mechanisms, cache and state slots, scheduler, loading, entry points."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import lisunex_cases as cases
import lisunex_oracle as oracle
from kotodama_b200.models.lisunex import LisunexConfig, LisunexModel
from kotodama_b200.models.registry import FAMILIES, load_model, read_config
from kotodama_b200.ops import get_ops
from kotodama_b200.serve.cache import HybridCache
from kotodama_b200.serve.engine import SamplingParams
from test_vunitar_cpu import write_model

ROOT = Path(__file__).resolve().parents[1]
F32 = torch.float32


def test_row_operations():
    cases.check_row_ops(get_ops("cpu"), "cpu", F32)


def test_rotary_positions_and_unit_heads():
    cases.check_rotary(get_ops("cpu"), "cpu", F32)


@pytest.mark.parametrize("case", cases.ATTENTION_CASES, ids=str)
def test_attention_at_chunk_borders_and_far_keys(case):
    cases.check_attention(get_ops("cpu"), "cpu", F32, *case)


@pytest.mark.parametrize("case", cases.DELTA_CASES, ids=str)
def test_delta_rule(case):
    cases.check_delta(get_ops("cpu"), "cpu", F32, *case)


def test_a_planted_mistake_shows():
    """The plain implementation with a key one chunk too far, without the pass vectors, with a forgotten state: each differs."""
    cfg = cases.CONFIGS["fit"]
    model = cases.weights(cfg, 2, (-7.0, 1.0))
    toks = cases.tokens(cfg, 120, 3)
    w = {k: v.double() for k, v in model.weights.items()}
    want = oracle.forward(cfg, w, toks)
    chunk = json.loads(json.dumps(cfg))
    chunk["layers"][1]["mixer"]["mask"]["size"] = 49
    nostep = {**w, "loop.step": torch.zeros_like(w["loop.step"])}
    for other in (oracle.forward(chunk, w, toks), oracle.forward(cfg, nostep, toks)):
        assert float(cases.row_errors(other, want).max()) > 0.2
    late = oracle.forward(cfg, w, toks[60:])           # the second half without what the first half left
    assert float(cases.row_errors(late, want[60:]).min()) > 0.05


@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_prompts_portions_and_decoding(name):
    cases.check_portions(name, "cpu", F32, lengths=(1, 2, 50, 110))


def test_batches_and_slots_used_again():
    cases.check_batches("odd", "cpu", F32)


def test_pages_behind_the_chunk_are_given_back():
    cases.check_pages_behind_the_chunk("fit", "cpu", F32)


def test_long_decoding():
    cases.check_long_decoding("odd", "cpu", F32, n=160)


def test_greedy_generation_through_the_scheduler():
    cases.check_generation("odd", "cpu", F32)
    cases.check_generation("one", "cpu", F32)


def test_passes_of_the_loop_have_their_own_cache_and_state():
    cfg = cases.CONFIGS["odd"]
    eng = cases.engine(cases.weights(cfg), "cpu", F32, max_ctx=64)
    assert eng.runner.runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert [k is not None for k in eng.cache.k] == [i in (1, 3) for i, _ in eng.runner.runs]
    assert [s is not None for s in eng.cache.state] == [i in (0, 2) for i, _ in eng.runner.runs]
    s = eng.open()
    eng.feed([(s, cases.tokens(cfg, 30, 0), [])])
    kept = [k for k in eng.cache.k if k is not None and k.shape == eng.cache.k[1].shape]
    assert all(not torch.equal(a, b) for i, a in enumerate(kept) for b in kept[:i])


def test_state_slots():
    cfg = cases.CONFIGS["one"]
    eng = cases.engine(cases.weights(cfg), "cpu", F32, max_ctx=32, max_batch=2)
    seqs = [eng.open() for _ in range(3)]
    for s in seqs[:2]:
        eng.feed([(s, [1, 2], [])])
    with pytest.raises(RuntimeError):
        eng.feed([(seqs[2], [1], [])])
    eng.close(seqs[0])
    eng.feed([(seqs[2], [1], [])])
    assert seqs[2].state >= 0 and seqs[2].state != seqs[1].state
    # families without recurrent layers have none
    plain = HybridCache([(1, 8, 8)], [None], 2, 4, torch.device("cpu"), F32)
    assert plain.num_states == 0 and plain.can_take_state() and plain.take_state() == -1


def test_requests_wait_for_slots_and_cancel_returns_them():
    cfg = cases.CONFIGS["fit"]
    model = cases.weights(cfg)
    eng = cases.engine(model, "cpu", F32, max_ctx=96, max_batch=2, prefill_portion=8)
    short = eng.add_request(cases.tokens(cfg, 4, 0), SamplingParams(max_new_tokens=12, temperature=0.0))
    long = eng.add_request(cases.tokens(cfg, 40, 1), SamplingParams(max_new_tokens=4, temperature=0.0))
    third = eng.add_request(cases.tokens(cfg, 6, 4), SamplingParams(max_new_tokens=3, temperature=0.0))
    eng.step()
    assert len(short.generated) == 2 and long.ctx_len == 8 and third.state < 0
    assert eng.cancel(long.rid)                                    # in the middle of its prompt
    while eng.has_work():
        eng.step()
    assert short.generated == cases.greedy(cfg, model, short.prompt, 12)
    assert third.generated == cases.greedy(cfg, model, third.prompt, 3)
    assert len(eng.cache.free) == eng.cache.num_pages and len(eng.cache.free_states) == 2


def test_sampled_generation_is_reproducible():
    cfg = cases.CONFIGS["fit"]
    eng = cases.engine(cases.weights(cfg), "cpu", F32, max_ctx=96)
    p = SamplingParams(max_new_tokens=10, temperature=0.8, top_k=20, top_p=0.9, repetition_penalty=1.2, seed=5)
    prompt = cases.tokens(cfg, 20, 0)
    a = eng.generate([prompt, prompt], p)
    assert a[0] == a[1] == eng.generate([prompt], p)[0] and len(set(a[0])) > 3


def test_model_folder_loads_by_architecture(tmp_path):
    cfg = cases.CONFIGS["odd"]
    model = cases.weights(cfg)
    folder = write_model(tmp_path / "m", cfg, model.weights)
    back = load_model(folder)
    assert isinstance(back, LisunexModel) and all(torch.equal(back.weights[k], v) for k, v in model.weights.items())
    assert back.config.param_count() == sum(v.numel() for v in model.weights.values())
    family, lc = read_config(folder)
    assert family is FAMILIES["Lisunex"] and lc.to_dict() == cfg
    assert isinstance(family.random(lc, 3), LisunexModel)


def test_wrong_weights_and_configurations_are_refused():
    cfg = cases.CONFIGS["odd"]
    w = dict(cases.weights(cfg).weights)
    lc = LisunexConfig.from_dict(cfg)
    with pytest.raises(KeyError):
        LisunexModel(lc, {k: v for k, v in w.items() if k != "loop.step"})
    with pytest.raises(ValueError):
        LisunexModel(lc, {**w, "l0.mix.q.conv": w["l0.mix.q.conv"][:, 1:]})
    first = cfg["layers"][0]
    for change in (dict(type="other"), dict(mlp=dict(kind="other")), dict(mixer=dict(first["mixer"], kv_heads=4))):
        with pytest.raises(ValueError):
            LisunexConfig.from_dict({**cfg, "layers": [{**first, **change}], "loop": None})
    for loop in ((2, 2, 1), (0, 5, 1), (0, 2, 0)):
        with pytest.raises(ValueError):
            LisunexConfig.from_dict({**cfg, "loop": dict(zip(("start", "stop", "times"), loop))})
    odd = json.loads(json.dumps(cfg))
    odd["layers"][1]["mixer"]["rot"]["dims"] = 30
    with pytest.raises(ValueError):
        LisunexConfig.from_dict(odd)


def test_trace_replay_program(tmp_path):
    cfg = cases.CONFIGS["odd"]
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

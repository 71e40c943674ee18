"""Sapasun through the framework's own entry points against the plain oracle: whole prompts, portions, decoding through the cache,
batches, reused blocks and slots, preemption, greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import sapasun_oracle as oracle
from busatar_oracle import write_model
from sapasun_configs import CONFIGS

TOL = {"f32": 4e-5, "bf16": 4e-2}


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# ------------------------------------------------------------------------------------------------ host side
def test_configuration_is_read_from_the_file(tmp_path):
    from openvino_b200.models.llm_config import PARALLEL_NORM, AttentionSpec, ChannelDeltaSpec, RotarySpec, SquaredReluSpec
    from openvino_b200.models.registry import from_dict, load_checkpoint
    cfg = CONFIGS["mixed"]
    weights = oracle.random_weights(cfg, 1)
    write_model(tmp_path, cfg, weights)
    ck = load_checkpoint(str(tmp_path))
    c = ck.config
    assert (c.name, c.vocab_size, c.hidden_size, c.norm_eps, c.norm_offset, c.block, c.embed_norm, c.logit_softcap) == \
        ("Sapasun", 320, 192, 1e-5, 0.0, PARALLEL_NORM, True, 9.0)
    assert [type(l.mixer) for l in c.layers] == [AttentionSpec, ChannelDeltaSpec, AttentionSpec, ChannelDeltaSpec, AttentionSpec, AttentionSpec]
    assert c.layers[2].mlp is None and c.layers[1].mlp == SquaredReluSpec(128) and c.has_recurrent_state
    assert c.layers[1].mixer == ChannelDeltaSpec(6, 2, 32, 48, 4)
    assert c.layers[2].mixer == AttentionSpec(6, 2, 48, 32, 0.4, rotary=RotarySpec(24, 500.0), head_gate=True, chunk=33, sink=True, taps=2, v_mix=True)
    assert not c.layers[0].mixer.v_mix and c.layers[5].mixer.taps == 1 and not c.layers[5].mixer.carries_state
    shapes = ck.arch.tensor_shapes(c)
    assert set(shapes) == set(weights)
    for n, t in weights.items():
        assert len(shapes[n]) == t.dim() and all(w in (None, s) for w, s in zip(shapes[n], t.shape)), n
        assert torch.equal(ck.tensors[n].float(), t)
    assert torch.equal(ck(1, "mix", "a2").float(), weights["l1.mix.a2"]) and ck(2, "mix", "vmix").dim() == 0
    wrong = dict(weights, **{"l1.mix.a2": weights["l1.mix.a2"][:-1]})
    with pytest.raises(ValueError, match="'l1.mix.a2' has the shape"):
        from_dict(cfg, wrong)(1, "mix", "a2")
    for path, value, what in (("type", "mamba", "token mixer"), ("mlp", {"kind": "moe"}, "feed-forward")):
        bad = json.loads(json.dumps(cfg))
        bad["layers"][0][path] = value
        with pytest.raises(ValueError, match=what):
            from_dict(bad, weights)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["mixer"]["kv_heads"] = 4
    with pytest.raises(ValueError, match="evenly"):
        from_dict(bad, weights)


def test_only_models_with_state_refuse_prefix_caching():
    from openvino_b200.models.registry import from_dict
    assert from_dict(CONFIGS["recurrent"], {}).config.has_recurrent_state
    assert from_dict(CONFIGS["attention"], {}).config.has_recurrent_state           # inputs of the second layer's filters
    one_tap = dict(CONFIGS["attention"], layers=CONFIGS["attention"]["layers"][:1])
    assert not from_dict(one_tap, {}).config.has_recurrent_state


def test_oracle_decodes_as_it_reads_whole_sequences():
    """The oracle has no cache: its logits at a position must not change when the sequence goes on."""
    cfg = CONFIGS["odd"]
    w, ids = oracle.random_weights(cfg, 3), tokens(44, 131, 1)
    full = oracle.forward(cfg, w, ids)[0]
    for n in (1, 2, 7, 8, 21, 22, 43):
        assert torch.allclose(oracle.forward(cfg, w, ids[:n])[0], full[:n], atol=1e-9)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_every_tensor_matters(name):
    """A weight that did not show in the logits would not be tested by the comparisons below (the first mixing layer's own factor is
    the one that is not used)."""
    cfg = CONFIGS[name]
    w, ids = oracle.random_weights(cfg, 7), tokens(45, cfg["vocab"], 2)
    base = oracle.forward(cfg, w, ids)[0]
    mixing = [i for i, l in enumerate(cfg["layers"]) if l["type"] == "attention" and l["mixer"]["v_mix"]]
    for key in w:
        changed = dict(w, **{key: w[key] * 1.5 + 0.1})
        d = (oracle.forward(cfg, changed, ids)[0] - base).abs().max() / base.std()
        unused = key.endswith(".vmix") and int(key[1:].split(".")[0]) not in mixing[1:]
        assert (d == 0) if unused else (d > 1e-2), (key, float(d))


# ------------------------------------------------------------------------------------------------ on the GPU
_cache = {}


def model(name):
    if name not in _cache:
        cfg = CONFIGS[name]
        _cache[name] = (cfg, oracle.random_weights(cfg, 7))
    return _cache[name]


def want_logits(name, ids):
    key = (name, tuple(ids))
    if key not in _cache:
        cfg, w = model(name)
        _cache[key] = oracle.forward(cfg, w, ids)[0]
    return _cache[key]


def replay(name, precision, max_tokens=512, seqs=8, **kw):
    from openvino_b200.genai.replay import Replay
    from openvino_b200.models.registry import from_dict
    from openvino_b200.runtime.layered_llm import create_executor
    cfg, w = model(name)
    ex, _ = create_executor(from_dict(cfg, {k: v.to(torch.bfloat16) for k, v in w.items()}), max_num_seqs=seqs, max_num_batched_tokens=max_tokens,
                            max_model_len=max_tokens, properties={"INFERENCE_PRECISION_HINT": precision}, **kw)
    return Replay(ex)


def compare(got, want, precision):
    got, want = got.double(), want.double()
    d = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert torch.isfinite(d).all() and d.max() < TOL[precision], (int(d.argmax()), float(d.max()))


@pytest.mark.gpu
@pytest.mark.parametrize("precision", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompts_portions_and_decoding(name, precision):
    ids = tokens(300, CONFIGS[name]["vocab"], 5)
    want = want_logits(name, ids)
    r = replay(name, precision)
    every = lambda n: list(range(n))
    compare(r.step([("whole", ids, every(300))]), want, precision)
    for cut in (2, 3, 7, 64, 133):                             # portions of a prompt; the last one may be shorter
        got = [r.step([("cut%d" % cut, ids[i:i + cut], every(len(ids[i:i + cut])))]) for i in range(0, 300, cut)]
        compare(torch.cat(got), want, precision)
        r.end("cut%d" % cut)
    got = [r.step([("dec", ids[:1], [0])])] + [r.step([("dec", [t], [0])]) for t in ids[1:]]      # token by token from the first
    compare(torch.cat(got), want, precision)
    r.end("dec")
    got = [r.step([("long", ids[:129], every(129))])] + [r.step([("long", [t], [0])]) for t in ids[129:]]
    compare(torch.cat(got), want, precision)


@pytest.mark.gpu
@pytest.mark.parametrize("precision", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "large"])
def test_batches_do_not_mix_requests(name, precision):
    """Unequal requests in one batch, prompts beside decoding ones, blocks and slots that another request has just left."""
    V = CONFIGS[name]["vocab"]
    reqs = {k: tokens(n, V, i) for i, (k, n) in enumerate([("a", 90), ("b", 1), ("c", 33), ("d", 150), ("e", 64), ("f", 17)])}
    at = {k: 0 for k in reqs}
    r = replay(name, precision, max_tokens=256, seqs=4, kv_cache_blocks=16)      # no room for two long requests more than needed
    plan = [dict(a=40, b=1, c=20), dict(a=1, c=1), dict(a=2, c=3, d=60), dict(a=1, c=9, d=1), dict(a=46, d=2), dict(d=40, e=1), dict(d=1, e=30, f=16),
            dict(d=46, e=1, f=1), dict(e=32)]
    for step in plan:
        got = r.step([(k, reqs[k][at[k]:at[k] + n], list(range(n))) for k, n in step.items()])
        lo = 0
        for k, n in step.items():
            compare(got[lo:lo + n], want_logits(name, reqs[k])[at[k]:at[k] + n], precision)
            lo += n
            at[k] += n
            if at[k] == len(reqs[k]):
                r.end(k)
    assert all(at[k] == len(reqs[k]) for k in reqs) and r.scheduler.blocks.num_free() == 16


@pytest.mark.gpu
@pytest.mark.parametrize("precision", ["f32", "bf16"])
def test_steps_larger_than_the_executor_run_in_portions(precision):
    ids = tokens(150, 320, 2)
    r = replay("mixed", precision, max_tokens=64, seqs=2, kv_cache_blocks=64)
    got = r.step([("x", ids[:60], [59]), ("y", ids[:33], [0, 32]), ("z", ids[:5], [4])])
    compare(got, want_logits("mixed", ids)[[59, 0, 32, 4]], precision)


@pytest.mark.gpu
def test_long_decoding_crosses_many_chunks():
    """Seven hundred decoded tokens: every chunk size of the model begins anew many times, the recurrent state stays exact."""
    ids = tokens(720, 131, 12)
    want = want_logits("odd", ids)
    for precision in ("f32", "bf16"):
        r = replay("odd", precision, max_tokens=1024, seqs=2)
        got = [r.step([("x", ids[:20], [19])])] + [r.step([("x", [t], [0])]) for t in ids[20:]]
        compare(torch.cat(got), want[19:], precision)


def checkpoint(tmp_path, name):
    cfg, w = model(name)
    write_model(tmp_path, cfg, w)
    return str(tmp_path)


def follows_greedy(name, prompt, out, slack):
    """Every generated token is the oracle's best given what came before, or within ``slack`` of it."""
    lg = want_logits(name, prompt + out[:-1])[len(prompt) - 1:]
    for row, t in zip(lg, out):
        assert row[t] >= row.max() - slack * row.std(), (float(row.max() - row[t]), float(row.std()))


@pytest.mark.gpu
@pytest.mark.parametrize("precision,native", [("f32", True), ("bf16", True), ("bf16", False)])
@pytest.mark.parametrize("fuse", [False, True])
def test_greedy_generation_through_the_pipeline(tmp_path, precision, native, fuse):
    """More requests than slots, prompts longer than a step's budget, decoding past chunk borders, both schedulers."""
    from openvino_b200.genai import GenerationConfig, LLMPipeline
    from openvino_b200.genai.pipeline import ContinuousBatchingPipeline
    pipe = LLMPipeline(checkpoint(tmp_path, "mixed"), "CUDA", max_num_seqs=3, max_num_batched_tokens=48, max_model_len=256,
                       INFERENCE_PRECISION_HINT=precision, dynamic_split_fuse=fuse)
    if not native:
        pipe.scheduler_config.use_native = False
        pipe.pipeline = ContinuousBatchingPipeline(pipe.executor, pipe.scheduler_config)
    prompts = [tokens(n, 320, 100 + n) for n in (5, 70, 1, 33, 111)]
    outs = pipe.generate(prompts, GenerationConfig(max_new_tokens=60))
    for p, o in zip(prompts, outs):
        assert len(o) == 60
        follows_greedy("mixed", p, o, 1e-4 if precision == "f32" else 0.1)
    assert pipe.pipeline.metrics.preemptions == 0
    again = pipe.generate(prompts[:2], GenerationConfig(max_new_tokens=60))          # used slots and blocks
    if precision == "f32":
        assert again == outs[:2]


@pytest.mark.gpu
@pytest.mark.parametrize("native", [True, False])
def test_preempted_requests_start_over(tmp_path, native):
    from openvino_b200.genai import GenerationConfig, LLMPipeline
    from openvino_b200.genai.pipeline import ContinuousBatchingPipeline
    pipe = LLMPipeline(checkpoint(tmp_path, "mixed"), "CUDA", max_num_seqs=4, max_num_batched_tokens=64, max_model_len=128, kv_cache_blocks=14,
                       INFERENCE_PRECISION_HINT="f32")
    pipe.scheduler_config.use_native = native
    pipe.pipeline = ContinuousBatchingPipeline(pipe.executor, pipe.scheduler_config)
    prompts = [tokens(n, 320, 200 + n) for n in (40, 50, 45, 30)]
    outs = pipe.generate(prompts, GenerationConfig(max_new_tokens=50))
    assert pipe.pipeline.metrics.preemptions > 0
    for p, o in zip(prompts, outs):
        follows_greedy("mixed", p, o, 1e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["recurrent", "mixed"])
def test_decode_graphs_leave_the_state_alone(name):
    """Capturing a decode step runs it once for warm-up; neither recurrent state nor the inputs of filters may advance twice."""
    ids = tokens(40, CONFIGS[name]["vocab"], 8)
    r = replay(name, "f32")
    r.step([("x", ids[:20], [])])
    assert not r.ex._graphs
    got = torch.cat([r.step([("x", [t], [0])]) for t in ids[20:]])
    assert r.ex._graphs
    compare(got, want_logits(name, ids)[20:], "f32")


@pytest.mark.gpu
def test_sampling_and_command_line(tmp_path):
    from openvino_b200.genai import GenerationConfig, LLMPipeline
    path = checkpoint(tmp_path, "recurrent")
    pipe = LLMPipeline(path, "CUDA", max_num_seqs=4, max_num_batched_tokens=64, max_model_len=128, INFERENCE_PRECISION_HINT="f32")
    prompt = tokens(20, 96, 20)
    out = pipe.generate(prompt, GenerationConfig(max_new_tokens=20, do_sample=True, temperature=0.8, top_k=20, top_p=0.9, rng_seed=3))
    assert len(out) == 20 and all(0 <= t < 96 for t in out)
    assert pipe.generate(prompt, GenerationConfig(max_new_tokens=9, do_sample=True, temperature=1.0, top_k=1, rng_seed=1)) == \
        pipe.generate(prompt, GenerationConfig(max_new_tokens=9))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    run = subprocess.run([sys.executable, os.path.join(root, "samples", "python", "llm_generate.py"), path, "ids:" + ",".join(map(str, prompt))],
                         capture_output=True, text=True, timeout=300, env=dict(os.environ, PYTHONPATH=root))
    assert run.returncode == 0, run.stderr[-2000:]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_command(tmp_path, dtype):
    path = checkpoint(tmp_path / "m", "odd")
    out = tmp_path / "out"
    out.mkdir()
    ids = [tokens(30, 131, 1), tokens(50, 131, 2)]
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": ids[0][:20], "want": [0, 19]}, {"id": "q", "tokens": ids[1][:41], "want": [40]}], "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": ids[0][20:21], "want": []}, {"id": "q", "tokens": ids[1][41:42], "want": []}], "end": ["p"]},
             {"step": 2, "entries": [{"id": "q", "tokens": ids[1][42:43], "want": [0]}], "end": ["q"]},
             {"step": 3, "entries": [{"id": "p", "tokens": ids[0], "want": [29]}], "end": ["p"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    run = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == ["done %d" % i for i in range(4)]
    read = lambda i: torch.from_numpy(np.fromfile(out / ("%d.f32" % i), dtype="<f4").reshape(-1, 131).copy())
    w = [want_logits("odd", x) for x in ids]
    p = "f32" if dtype == "float32" else "bf16"
    compare(read(0), torch.stack([w[0][0], w[0][19], w[1][40]]), p)
    compare(read(2), w[1][42:43], p)
    compare(read(3), w[0][29:30], p)

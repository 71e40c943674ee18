"""Busatar through the framework's own entry points against the plain oracle: whole prompts, portions, decoding through the cache,
batches, reused blocks and slots, preemption, greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import busatar_oracle as oracle
from busatar_configs import CONFIGS

TOL = {"f32": 3e-5, "bf16": 3e-2}


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# ------------------------------------------------------------------------------------------------ host side
def test_configuration_is_read_from_the_file(tmp_path):
    from openvino_b200.models.llm_config import AttentionSpec, LatentAttentionSpec, LimitedGluSpec, RgLruSpec
    from openvino_b200.models.registry import from_dict, load_checkpoint
    cfg = CONFIGS["mixed"]
    weights = oracle.random_weights(cfg, 1)
    oracle.write_model(tmp_path, cfg, weights)
    ck = load_checkpoint(str(tmp_path))
    c = ck.config
    assert (c.vocab_size, c.hidden_size, c.residual_scale, c.norm_eps, c.norm_offset) == (320, 192, 1.7, 1e-5, 1.0)
    assert [type(l.mixer) for l in c.layers] == [LatentAttentionSpec, AttentionSpec, RgLruSpec, LatentAttentionSpec, RgLruSpec, AttentionSpec]
    assert c.layers[1].mlp is None and c.layers[2].mlp == LimitedGluSpec(192, 0.8) and c.has_recurrent_state
    assert c.layers[1].mixer == AttentionSpec(6, 2, 48, 32, 0.5, 33, qk_norm=True, gated=True)
    assert c.layers[2].mixer == RgLruSpec(160, 5, 4)
    m = c.layers[0].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window, m.scale) == (4, 32, 8, 48, 64, 40, 0.3)
    for name, t in weights.items():
        assert torch.equal(ck.tensors[name].float(), t)
    assert torch.equal(ck(2, "mix", "conv").float(), weights["l2.mix.conv"]) and torch.equal(ck(-1, "", "head").float(), weights["head"])
    with pytest.raises(KeyError, match="no tensor 'l9.mix.q'"):
        ck(9, "mix", "q")
    assert ck.arch.tensor_shapes(c) == {n: tuple(t.shape) for n, t in weights.items()}
    wrong = dict(weights, head=weights["head"][:-1])
    with pytest.raises(ValueError, match="'head' has the shape"):
        from_dict(cfg, wrong)(-1, "", "head")
    with pytest.raises(ValueError, match="unknown architecture"):
        (tmp_path / "config.json").write_text(json.dumps(dict(cfg, architecture="Nobody")))
        load_checkpoint(str(tmp_path))


def test_safetensors_reader_refuses_damaged_files(tmp_path):
    from openvino_b200.utils.safetensors import SafetensorsFile
    oracle.write_model(tmp_path, {}, {"a": torch.ones(3, 4), "b": torch.zeros(0)})
    path = tmp_path / "model.safetensors"
    f = SafetensorsFile(str(path))
    assert f.keys() == ["a", "b"] and "a" in f and f.shape("a") == (3, 4) and f["b"].numel() == 0 and f["a"].dtype == torch.bfloat16
    path.write_bytes(path.read_bytes()[:-2])
    with pytest.raises(ValueError, match="does not fit"):
        SafetensorsFile(str(path))["a"]
    path.write_bytes(b"\xff" * 16)
    with pytest.raises(ValueError, match="header"):
        SafetensorsFile(str(path))


@pytest.mark.parametrize("rot", [dict(dims=16, base=1e6, scaling=dict(factor=2.0, original=2048, fast=32.0, slow=1.0)), dict(dims=64, base=1e4),
                                 dict(dims=64, base=1e4, scaling=dict(factor=40.0, original=4096, fast=32.0, slow=1.0)),
                                 dict(dims=8, base=500.0, scaling=dict(factor=3.0, original=16, fast=4.0, slow=4.0))])
def test_rotary_frequencies(rot):
    from openvino_b200.models.busatar import _rotary
    spec = _rotary(rot)
    f, mult = oracle.yarn(rot)
    assert np.allclose(spec.inv_freq(), f.numpy(), rtol=1e-12) and abs(spec.multiplier() - mult) < 1e-12


@pytest.mark.parametrize("native", [True, False])
def test_descriptor_carries_state_slots(native):
    from openvino_b200.genai.native_scheduler import NativeScheduler, make_layout
    from openvino_b200.genai.scheduler import Scheduler, SchedulerConfig, Sequence
    cfg = SchedulerConfig(max_num_batched_tokens=8, max_num_seqs=4, num_kv_blocks=32, block_size=4)
    offs, off = {}, 0
    for name, n in (("ids", 8), ("positions", 8), ("slot_map", 8), ("tok_src", 8), ("tok_dst", 4), ("logit_idx", 4), ("past_lens", 4), ("subsequence_begins", 5),
                    ("block_indices_begins", 5), ("block_indices", 32), ("state_slots", 4)):
        offs[name] = (off, n)
        off += n
    s = NativeScheduler(cfg) if native else Scheduler(cfg)
    for i, n in enumerate((3, 11, 2)):
        s.add(Sequence(i, np.arange(n, dtype=np.int32), 3))
    seen = {}
    while s.has_unfinished():
        st = s.schedule()
        d = np.full(off, -7, dtype=np.int32)
        if native:
            s.fill_flat(st, d, make_layout(offs, 8, 4, 8))
        else:
            s.fill(st, {k: d[o:o + n] for k, (o, n) in offs.items()})
        got = d[offs["state_slots"][0]:][:len(st.seqs)].tolist()
        assert len(set(got)) == len(got) and all(0 <= x < 16 for x in got)
        for q, x in zip(st.seqs, got):          # a prompt in portions (where tok_dst is still -1) keeps its slot
            assert seen.setdefault(q.request_id, x) == x
        s.commit(st, np.zeros(8, dtype=np.int32))


def test_prefix_caching_is_refused_with_recurrent_state():
    from openvino_b200.genai.pipeline import ContinuousBatchingPipeline
    from openvino_b200.genai.scheduler import SchedulerConfig

    class Recurrent:
        has_recurrent_state = True
    with pytest.raises(ValueError, match="prefix caching"):
        ContinuousBatchingPipeline(Recurrent(), SchedulerConfig(enable_prefix_caching=True))


def test_oracle_decodes_as_it_reads_whole_sequences():
    """The oracle has no cache: its logits at a position must not change when the sequence goes on."""
    cfg = CONFIGS["odd"]
    w, ids = oracle.random_weights(cfg, 3), tokens(40, 131, 1)
    full = oracle.forward(cfg, w, ids)[0]
    for n in (1, 2, 21, 22, 39):
        assert torch.allclose(oracle.forward(cfg, w, ids[:n])[0], full[:n], atol=1e-9)


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


def compare(got, want, precision, tol=None):
    got, want = got.double(), want.double()
    d = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert torch.isfinite(d).all() and d.max() < (tol or TOL[precision]), (int(d.argmax()), float(d.max()))


@pytest.mark.gpu
@pytest.mark.parametrize("precision", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompts_portions_and_decoding(name, precision):
    ids = tokens(300, CONFIGS[name]["vocab"], 5)
    want = want_logits(name, ids)
    r = replay(name, precision)
    every = lambda n: list(range(n))
    compare(r.step([("whole", ids, every(300))]), want, precision)
    for cut in (2, 7, 64, 133):                                # portions of a prompt; the last one may be shorter
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
    slots = set()
    plan = [dict(a=40, b=1, c=20), dict(a=1, c=1), dict(a=2, c=3, d=60), dict(a=1, c=9, d=1), dict(a=46, d=2), dict(d=40, e=1), dict(d=1, e=30, f=16),
            dict(d=46, e=1, f=1), dict(e=32)]
    for step in plan:
        entries = [(k, reqs[k][at[k]:at[k] + n], list(range(n))) for k, n in step.items()]
        got = r.step(entries)
        lo = 0
        for k, n in step.items():
            compare(got[lo:lo + n], want_logits(name, reqs[k])[at[k]:at[k] + n], precision)
            slots.add((k, r.requests[k].slot))
            lo += n
            at[k] += n
            if at[k] == len(reqs[k]):
                r.end(k)
    assert all(at[k] == len(reqs[k]) for k in reqs) and r.scheduler.blocks.num_free() == 16
    with pytest.raises(RuntimeError, match="too small"):
        r.step([("huge", tokens(16 * 16 + 1, V, 9)[:256], []), ("more", [1], [])])


@pytest.mark.gpu
@pytest.mark.parametrize("precision", ["f32", "bf16"])
def test_steps_larger_than_the_executor_run_in_portions(precision):
    ids = tokens(150, 320, 2)
    r = replay("mixed", precision, max_tokens=64, seqs=2, kv_cache_blocks=64)
    got = r.step([("x", ids[:60], [59]), ("y", ids[:33], [0, 32]), ("z", ids[:5], [4])])
    w = want_logits("mixed", ids)
    compare(got, w[[59, 0, 32, 4]], precision)


def checkpoint(tmp_path, name):
    cfg, w = model(name)
    oracle.write_model(tmp_path, cfg, w)
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
    """More requests than slots, prompts longer than a step's budget, decoding past every window, both schedulers."""
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
def test_sampling_and_staged_plans(tmp_path):
    from openvino_b200.genai import GenerationConfig, LLMPipeline
    pipe = LLMPipeline(checkpoint(tmp_path, "recurrent"), "CUDA", max_num_seqs=4, max_num_batched_tokens=64, max_model_len=128)
    prompts = [tokens(n, 96, n) for n in (20, 3)]
    a = pipe.generate(prompts, GenerationConfig(max_new_tokens=20, do_sample=True, temperature=0.8, top_k=20, top_p=0.9, rng_seed=3))
    assert all(len(o) == 20 and all(0 <= t < 96 for t in o) for o in a)
    greedy = pipe.generate(prompts, GenerationConfig(max_new_tokens=12))
    ex = pipe.executor
    pipe.pipeline.run_plan(pipe.pipeline.plan(prompts, GenerationConfig(max_new_tokens=12, ignore_eos=True)))
    torch.cuda.synchronize()
    assert sorted(ex.decode.tokens[:2].tolist()) == sorted(o[-1] for o in greedy)
    assert ex.kernel_launches > 0 and ex.kv_cache_bytes() > 0


@pytest.mark.gpu
def test_decode_graphs_leave_the_state_alone():
    """Capturing a decode step runs it once for warm-up; the recurrent state must not advance twice."""
    ids = tokens(40, 96, 8)
    want = want_logits("recurrent", ids)
    r = replay("recurrent", "f32")
    r.step([("x", ids[:20], [])])
    assert not r.ex._graphs
    got = torch.cat([r.step([("x", [t], [0])]) for t in ids[20:]])
    assert r.ex._graphs
    compare(got, want[20:], "f32")


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
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
    read = lambda i: torch.from_numpy(np.fromfile(out / ("%d.f32" % i), dtype="<f4").reshape(-1, 131).copy())
    w = [want_logits("odd", x) for x in ids]
    p = "f32" if dtype == "float32" else "bf16"
    compare(read(0), torch.stack([w[0][0], w[0][19], w[1][40]]), p)
    compare(read(2), w[1][42:43], p)
    compare(read(3), w[0][29:30], p)

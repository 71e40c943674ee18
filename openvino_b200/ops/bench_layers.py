"""Prefill and decode throughput of layered decoders beside the closest other model at equal size (random weights, bf16), and the
device time of every kernel call of a step with its roofline fraction: Busatar beside the Llama-family program, Sapasun beside Busatar.

    python bench.py --model busatar [--kernels] [--sizes gqa-4k,latent-4k]
    python bench.py --model sapasun [--kernels] [--sizes chunked-4k,delta-4k]

Both programs run through their executors: a prefill step is launched as the scheduler would (ragged batch, paged cache), a decode
step is replayed as its CUDA graph. Weights of a few layers exceed the L2 many times over. ``--kernels`` wraps every kernel entry
point with CUDA events and an L2 flush before the call; "like" kernels of the two programs have the same name in the table.
"""
from __future__ import annotations

from collections import OrderedDict
from typing import Dict, List, Tuple

import torch

from ..models.llm_config import (PARALLEL_NORM, AttentionSpec, ChannelDeltaSpec, LatentAttentionSpec, LayeredConfig, LayerSpec, LimitedGluSpec, LlmConfig, RgLruSpec,
                                 RotarySpec, SquaredReluSpec)
from ..models.registry import ARCHITECTURES, Checkpoint
from ..runtime.cuda_llm import CudaLlmExecutor, LlmWeights
from ..runtime.layered_llm import LayeredExecutor, LayeredWeights
from . import cuda as K
from .bench_kernels import _peaks


def _layered(width: int, mixers, ff: int, vocab: int = 32000) -> LayeredConfig:
    layers = tuple(LayerSpec(m, LimitedGluSpec(ff, 7.0) if mlp else None) for m, mlp in mixers)
    return LayeredConfig("Busatar", vocab, width, layers, residual_scale=2.0, norm_offset=1.0)


def _latent(heads, window):
    return LatentAttentionSpec(heads, 128, 64, 128, 512, 192 ** -0.5, RotarySpec(64, 10000.0, (8.0, 4096.0, 32.0, 1.0)), window)


def _gqa(heads, kv, window):
    return AttentionSpec(heads, kv, 128, 128, 128 ** -0.5, window, qk_norm=True, gated=True)


def _llama(width, heads, kv, ff, layers, window):
    return LlmConfig("llama-like", 32000, width, layers, heads, kv, 128, ff, weight_format="bf16", sliding_window=window)


# name -> (layered decoder, Llama of the same width, heads, feed-forward, window and number of layers)
SIZES: Dict[str, Tuple[LayeredConfig, LlmConfig]] = OrderedDict([
    ("gqa-4k", (_layered(4096, [(_gqa(32, 8, 4096), True)] * 4, 14336), _llama(4096, 32, 8, 14336, 4, 4096))),
    ("latent-4k", (_layered(4096, [(_latent(32, 4096), True)] * 4, 14336), _llama(4096, 32, 8, 14336, 4, 4096))),
    ("rglru-4k", (_layered(4096, [(RgLruSpec(4096, 16, 4), True)] * 4, 14336), _llama(4096, 32, 8, 14336, 4, 4096))),
    ("mixed-2k", (_layered(2048, [(_gqa(16, 4, 1024), True), (RgLruSpec(2560, 10, 4), False), (_latent(16, 1024), True), (_latent(16, 1024), True),
                                  (RgLruSpec(2560, 10, 4), True), (_gqa(16, 4, 1024), True)], 8192), _llama(2048, 16, 4, 8192, 6, 1024))),
])


def _parallel(width: int, mixers, ff: int, vocab: int = 32000) -> LayeredConfig:
    layers = tuple(LayerSpec(m, SquaredReluSpec(ff) if mlp else None) for m, mlp in mixers)
    return LayeredConfig("Sapasun", vocab, width, layers, block=PARALLEL_NORM, embed_norm=True, logit_softcap=30.0)


def _chunked(heads, kv, chunk):
    return AttentionSpec(heads, kv, 128, 128, 128 ** -0.5, rotary=RotarySpec(64, 10000.0), head_gate=True, chunk=chunk, sink=True, taps=4, v_mix=True)


def _delta(heads):
    return ChannelDeltaSpec(heads, heads, 128, 128, 4, decay_rank=128, gate_rank=128)


# name -> (Sapasun, Busatar of the same width, heads, window, layers and feed-forward parameters: a gated one has two input matrices)
SAPASUN_SIZES: Dict[str, Tuple[LayeredConfig, LayeredConfig]] = OrderedDict([
    ("chunked-4k", (_parallel(4096, [(_chunked(32, 8, 4096), True)] * 4, 21504), SIZES["gqa-4k"][0])),
    ("delta-4k", (_parallel(4096, [(_delta(32), True)] * 4, 21504), SIZES["rglru-4k"][0])),
    ("mixed-2k", (_parallel(2048, [(_chunked(16, 4, 1024), True), (_delta(16), False), (_chunked(16, 4, 1024), True), (_chunked(16, 4, 1024), True),
                                   (_delta(16), True), (_chunked(16, 4, 1024), True)], 12288), SIZES["mixed-2k"][0])),
])


class _RandomTensors:
    """Random tensors of a checkpoint's shapes, made on the device when they are asked for."""

    def __init__(self, shapes):
        self.shapes, self.g = shapes, torch.Generator(device="cuda").manual_seed(0)

    def __getitem__(self, name):
        shape = self.shapes[name]
        t = torch.randn(shape, device="cuda", generator=self.g)
        if name.endswith(".lam") or name.endswith(".dt_bias"):
            return (t - 3.0).to(torch.bfloat16)
        if len(shape) == 0:
            return torch.tensor(0.5, dtype=torch.bfloat16, device="cuda")
        if len(shape) == 1:
            return (1.0 + 0.1 * t if name.endswith("q.norm") or name.endswith("k.norm") or name.endswith("dkv.norm") else 0.1 * t).to(torch.bfloat16)
        return (t * shape[-1] ** -0.5).to(torch.bfloat16)


def make_layered(cfg: LayeredConfig, **kw) -> LayeredExecutor:
    arch = ARCHITECTURES[cfg.name]
    return LayeredExecutor(LayeredWeights(Checkpoint(cfg, arch, _RandomTensors(arch.tensor_shapes(cfg))), torch.device("cuda")), **kw)


class _Driver:
    """Steps of given batches on any executor: block tables and descriptors from the scheduler's own block manager."""

    def __init__(self, ex):
        from ..genai.scheduler import Scheduler, SchedulerConfig
        self.ex = ex
        self.sched = Scheduler(SchedulerConfig(max_num_batched_tokens=ex.prefill.Tcap, max_num_seqs=ex.max_seqs, num_kv_blocks=ex.num_kv_blocks,
                                               block_size=ex.block_size))
        self.g = torch.Generator().manual_seed(1)

    def start(self, lens: List[int]):
        import numpy as np
        from ..genai.scheduler import Sequence
        seqs = [Sequence(i, torch.randint(0, self.ex.cfg.vocab_size, (n,), generator=self.g).numpy().astype(np.int32), 0) for i, n in enumerate(lens)]
        for s in seqs:
            self.sched.admit(s)
        return seqs

    def stop(self, seqs):
        for s in seqs:
            self.sched.retire(s)

    def place(self, seqs, counts):
        from ..genai.pipeline import step_shape
        ex, st = self.ex, self.sched.place(seqs, counts)
        sb = ex.decode if st.max_q_len == 1 and len(seqs) <= ex.decode.Bcap else ex.prefill
        self.sched.fill(st, {n: sb.view(n, host=0).numpy() for n in sb.offsets})
        ex.upload(sb, 0)
        return st, sb, step_shape(st)

    def fill(self, seqs):
        """Run all known tokens but the last through the model."""
        while True:
            todo = [(s, min(len(s.prompt) - 1 - s.num_computed, self.ex.prefill.Tcap)) for s in seqs]
            batch, left = [], self.ex.prefill.Tcap
            for s, n in todo:
                n = min(n, left)
                if n > 0:
                    batch.append((s, n))
                    left -= n
            if not batch:
                return
            st, sb, shp = self.place([s for s, _ in batch], [n for _, n in batch])
            self.ex._forward(sb, shp)
            torch.cuda.synchronize()
            self.sched.advance(st)


def _time(fn, iters: int, warmup: int) -> float:
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


PREFILL = [(8, 1024), (1, 8192)]        # sequences x tokens of one step
DECODE = [(64, 2048), (1, 2048)]        # sequences x context


def run(executor, steps: int, warmup: int, kernels: bool) -> dict:
    d, out = _Driver(executor), {}
    with torch.no_grad():
        for B, n in PREFILL:
            seqs = d.start([n] * B)
            st, sb, shp = d.place(seqs, [n] * B)
            ms = _time(lambda: executor.run(sb, shp), steps, warmup)
            out["prefill %dx%d" % (B, n)] = {"ms": ms, "tokens_per_s": B * n / ms * 1e3}
            if kernels and B > 1:
                out["prefill %dx%d" % (B, n)]["kernels"] = profile(executor, lambda: executor._forward(sb, shp), [(0, n)] * B)
            d.stop(seqs)
        for B, n in DECODE:
            seqs = d.start([n] * B)
            d.fill(seqs)
            st, sb, shp = d.place(seqs, [1] * B)
            ms = _time(lambda: executor.run(sb, shp), 8 * steps, warmup)
            out["decode %dx%d" % (B, n)] = {"ms": ms, "tokens_per_s": B / ms * 1e3}
            if kernels and B > 1:
                out["decode %dx%d" % (B, n)]["kernels"] = profile(executor, lambda: executor._forward(sb, shp), [(n - 1, 1)] * B)
            d.stop(seqs)
    K.check_status("layer benchmark")
    return out


# ------------------------------------------------------------------------------------------------ kernels of a step
# fp32 arithmetic outside the tensor cores: 148 SMs x 128 multiply-adds a clock at 1.9 GHz (nominal)
FP32_TFLOPS = 148 * 128 * 2 * 1.9e-3


def _pairs(spans, window, chunk=0):
    """(query, key) pairs and distinct keys that a batch's tokens see."""
    pairs = keys = 0
    for past, new in spans:
        if chunk:
            pairs += sum(p % chunk + 1 for p in range(past, past + new))
            keys += past % chunk + new
            continue
        w = window or past + new
        pairs += sum(min(p + 1, w) for p in range(past, past + new))
        keys += min(past + new, new + w - 1)
    return pairs, keys


def _cost(name, args, kw, spans):
    """(label, bytes, flops on the tensor cores[, flops of fp32 arithmetic]) of a kernel call."""
    if name == "gemm":
        x, w = args[0], args[1]
        T, N = x.shape[0], w.N
        glu = kw.get("act", 0) in (K.ACT_SWIGLU, K.ACT_GLU_LIMITED)
        if kw.get("act", 0) in (K.ACT_RELU2, K.ACT_SOFTCAP):
            return "gemm N=%d K=%d +%s" % (N, w.K, "relu2" if kw["act"] == K.ACT_RELU2 else "softcap"), (N * w.K + T * w.K) * 2 + T * N * kw["out"].element_size(), \
                2.0 * T * N * w.K
        outb = T * N * (2 if glu is False and not kw.get("out_f32") else 4 if kw.get("out_f32") else 1)
        return "gemm N=%d K=%d%s" % (N, w.K, " +glu" if glu else ""), (N * w.K + T * w.K) * 2 + outb, 2.0 * T * N * w.K
    if name == "gemm_block_diag":
        x, w, out = args[:3]
        T = x.shape[0]
        return "block-diagonal gemm %dx%dx%d" % (w.G, w.N, w.K), w.G * (w.N * w.K * 2 + T * (w.K * 2 + w.N * out.element_size())), 2.0 * T * w.G * w.N * w.K
    if name in ("window_attention", "paged_attention"):
        if name == "paged_attention":
            Hq, Hkv, D = args[7:10]
            Dk = Dv = row = D
            T, latent, window, chunk = args[0].shape[0], False, kw["sliding_window"], 0
        else:
            Hq, Hkv, Dk, Dv, T, window = kw["Hq"], kw["Hkv"], kw["Dk"], kw["Dv"], kw["T"], kw["window"]
            latent, chunk = kw["k"] is kw["v"], kw.get("chunk", 0)
        pairs, keys = _pairs(spans, window, chunk)
        kv = keys * Hkv * (Dk if latent else Dk + Dv) * 2
        kind = "decode" if all(n == 1 for _, n in spans) else "prefill"
        return "%s attention %s" % ("latent" if latent else "paged", kind), kv + T * Hq * (Dk + Dv) * 2, 2.0 * pairs * Hq * (Dk + Dv)
    if name == "latent_prefill":
        pairs, keys = _pairs(spans, kw["window"])
        H, dk, dv = kw["H"], kw["k_head"] + kw["R"], kw["Dv"]
        return "paged attention prefill", (keys + kw["T"]) * H * (dk + dv) * 2, 2.0 * pairs * H * (dk + dv)
    if name == "latent_gather":
        return "latent gather", kw["rows"] * kw["cols"] * 4, 0.0
    if name == "rmsnorm":
        return "norm", args[0].numel() * 4, 0.0
    if name == "sum_rmsnorm":
        rows = (kw["row_idx"] if kw.get("row_idx") is not None else args[0]).shape[0]
        extra = [4 for key in ("y", "h_out", "s_out") if kw.get(key) is not None] + [2 for key in ("x_out", "x2_out") if kw.get(key) is not None]
        return "norm", rows * args[3] * (4 + sum(extra)), 0.0
    if name == "rope_kv_write":
        qkv, Hq, Hkv, D = args[0], args[5], args[6], args[7]
        return "head preparation", qkv.shape[0] * (Hq * 2 + Hkv * 4) * D * 2, 0.0
    if name == "heads_prepare":
        return "head preparation", kw["T"] * (kw["H"] * 2 * kw["D"] + kw["G"] * 2 * (kw["D"] + kw["Dv"])) * 2, 0.0
    if name == "channel_delta":
        # state: a decay (multiplication) and three multiply-adds per element and token, in fp32 by design
        T, H, G, dk, dv = kw["T"], kw["H"], kw["G"], kw["dk"], kw["dv"]
        return "recurrence", T * ((2 * G * dk + 2 * H * dv) * 2 + H * (dk + dv) * 4) + kw["B"] * H * dk * dv * 8, 0.0, 7.0 * T * H * dk * dv
    if name == "latent_prepare":
        return "head preparation (latent)", kw["T"] * (kw["H"] * 2 * kw["R"] + 2 * (kw["C"] + kw["R"])) * 2, 0.0
    if name == "causal_conv":
        return "short convolution", kw["T"] * kw["N"] * 4, 0.0
    if name == "lru_scan":
        return "recurrence", kw["T"] * kw["N"] * (8 + 2 + 2 + 2) + kw["B"] * kw["N"] * 8, 0.0
    return name, 0, 0.0


_NAMES = ("gemm", "gemm_block_diag", "window_attention", "paged_attention", "latent_prefill", "latent_gather", "rmsnorm", "sum_rmsnorm", "rope_kv_write",
          "heads_prepare", "latent_prepare", "causal_conv", "lru_scan", "channel_delta", "rope_table", "stream_embed", "embedding", "argmax", "resolve_ids", "scatter_tokens")


def profile(executor, step, spans, repeats: int = 3) -> List[dict]:
    """Every kernel call of ``step`` timed on its own (median over the calls of equal label), largest total first."""
    flush = torch.zeros(64 << 20, dtype=torch.int32, device="cuda")
    calls, saved = [], {n: getattr(K, n) for n in _NAMES}

    def wrap(name, fn):
        def timed(*args, **kw):
            label, nbytes, flops, *fp32 = _cost(name, args, kw, spans)
            flush.sum()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            out = fn(*args, **kw)
            b.record()
            calls.append((label, nbytes, flops, fp32[0] if fp32 else 0.0, a, b))
            return out
        return timed
    step()
    torch.cuda.synchronize()
    try:
        for n, fn in saved.items():
            setattr(K, n, wrap(n, fn))
        for _ in range(repeats):
            step()
    finally:
        for n, fn in saved.items():
            setattr(K, n, fn)
    torch.cuda.synchronize()
    groups: Dict[str, list] = OrderedDict()
    for label, nbytes, flops, fp32, a, b in calls:
        groups.setdefault(label, []).append((a.elapsed_time(b), nbytes, flops, fp32))
    peaks, rows = _peaks(), []
    for label, v in groups.items():
        ms, nbytes, flops, fp32 = sorted(v)[len(v) // 2]          # (calls of equal label may differ in size)
        us = ms * 1e3
        bounds = {"hbm": nbytes / (peaks["hbm_gbs"] * 1e3), "tensor": flops / (peaks["bf16_tflops"] * 1e6), "fp32": fp32 / (FP32_TFLOPS * 1e6)}
        kind = max(bounds, key=bounds.get)
        rows.append({"kernel": label, "calls": len(v) // repeats, "us": round(us, 1), "roofline_us": round(bounds[kind], 1),
                     "fraction": round(bounds[kind] / us, 3), "bound": kind})
    return sorted(rows, key=lambda r: -r["us"] * r["calls"])


def main(sizes: List[str], steps: int, warmup: int, kernels: bool, model: str = "busatar") -> dict:
    """Rows of the sizes that are named (all, if none is): {size: {model: ..., what it stands beside: ...}}."""
    rows, pairs = OrderedDict(), SAPASUN_SIZES if model == "sapasun" else SIZES
    for name in sizes or list(pairs):
        layered, other = pairs[name]
        limits = dict(num_kv_blocks=64 * (2048 // 16 + 2) + 64, block_size=16, max_batch_tokens=8192, max_seqs=64, max_blocks_per_seq=514)
        rows[name] = {}
        arms = ("sapasun", "busatar") if model == "sapasun" else ("layered", "llama")
        for arm, cfg in zip(arms, (layered, other)):
            if isinstance(cfg, LayeredConfig):
                ex = make_layered(cfg, **limits)
            else:
                ex = CudaLlmExecutor(cfg, LlmWeights.random(cfg, torch.device("cuda")), device="cuda", **limits)
            rows[name][arm] = run(ex, steps, warmup, kernels)
            del ex
            torch.cuda.empty_cache()
    return rows

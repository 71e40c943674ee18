"""Serving program of layered decoders (``LayeredConfig``): every layer is a token mixer and an optional feed-forward with sizes of
their own on an fp32 residual stream. Either each sum is followed by a norm (``POST_NORM``), or mixer and feed-forward read two norms of
the same stream and are added to it together (``PARALLEL_NORM``); their output projections are then one product over the concatenated
heads and activations.

The executor shares step descriptors, paging, CUDA graphs, sampling and token feedback with the other programs (``LlmExecutor``)
and adds per-layer caches: key / value pages of grouped-query attention, one row per token of latent attention, and fp32
recurrent state and inputs of short convolutions per request slot. Matrix products and activations are bf16 (fp32 accumulation), or everything is fp32 with
``dtype=torch.float32``.

Layout rules. Row pitches are multiples of 64 elements and heads are padded to 16, so that the tensor-core kernels read whole
fragments; weights carry zeros at the padding and every buffer starts out as zeros, so padding never contributes.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..models.llm_config import (PARALLEL_NORM, AttentionSpec, ChannelDeltaSpec, LatentAttentionSpec, LayeredConfig, LimitedGluSpec, RgLruSpec, RotarySpec,
                                 SquaredReluSpec)
from ..models.registry import Checkpoint
from ..ops import cuda as K
from .cuda_llm import LlmExecutor, StepBuffers, StepShape


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def _pad_rows(w: torch.Tensor, groups: int, pitch: int) -> torch.Tensor:
    """[groups * n, K] -> [groups * pitch, K] with zero rows behind every group's n."""
    n = w.shape[0] // groups
    return torch.nn.functional.pad(w.reshape(groups, n, -1), (0, 0, 0, pitch - n)).reshape(groups * pitch, -1)


def _pad_cols(w: torch.Tensor, groups: int, pitch: int) -> torch.Tensor:
    N, n = w.shape[0], w.shape[1] // groups
    return torch.nn.functional.pad(w.reshape(N, groups, n), (0, pitch - n)).reshape(N, groups * pitch)


class _Packer:
    """Checkpoint tensors of one layer -> device tensors in kernel layout, in the compute type."""

    def __init__(self, ckpt: Checkpoint, layer: int, device, dtype: torch.dtype):
        self.ckpt, self.layer, self.device, self.dtype = ckpt, layer, device, dtype

    def raw(self, part: str, key: str) -> torch.Tensor:
        return self.ckpt(self.layer, part, key).to(self.device)

    def f32(self, part: str, key: str, pad_to: int = 1) -> torch.Tensor:
        t = self.raw(part, key).float().reshape(-1)
        return torch.nn.functional.pad(t, (0, _up(t.numel(), pad_to) - t.numel())).contiguous()

    def linear(self, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> K.PackedWeight:
        """[N, K] with K padded to the pitch of its input."""
        w = torch.nn.functional.pad(w.to(self.dtype), (0, _up(w.shape[1], 64) - w.shape[1])).contiguous()
        bias = bias.to(self.dtype).contiguous() if bias is not None else None
        if self.dtype == torch.float32:
            return K.PackedWeight(K.W_F32, w, w.shape[0], w.shape[1], bias=bias)
        return K.PackedWeight.from_dense(w, bias=bias)

    def block_diag(self, w: torch.Tensor) -> K.BlockDiagWeight:
        return K.BlockDiagWeight(w.to(self.dtype).contiguous())


class _Rotation:
    def __init__(self, rot: Optional[RotarySpec], device):
        self.dims = rot.dims if rot else 0
        self.mult = rot.multiplier() if rot else 1.0
        self.freq = tuple(rot.inv_freq()) if rot else ()
        self.inv_freq = torch.tensor(self.freq, dtype=torch.float64).float().to(device) if rot else None

    def args(self) -> dict:
        return dict(rot_dims=self.dims, rot_mult=self.mult, inv_freq=self.inv_freq)


class _ShortConv:
    """Filters of short causal convolutions on the first columns of a projection, and the ring of inputs of every request slot."""

    def __init__(self, filters: List[torch.Tensor]):
        self.w = torch.cat([f.float() for f in filters], 0).t().contiguous()      # [taps, columns]
        self.taps, self.cols = self.w.shape

    def allocate(self, ex: "LayeredExecutor") -> None:
        self.ring = torch.zeros((ex.num_slots, self.taps, self.cols), dtype=torch.float32, device=ex.device)

    def args(self, sb: "LayeredStepBuffers", shp: StepShape) -> dict:
        return dict(conv_w=self.w, conv_ring=self.ring, conv_cols=self.cols, taps=self.taps, subsequence_begins=sb.view("subsequence_begins"),
                    past_lens=sb.view("past_lens"), slots=sb.view("state_slots"), B=shp.B, max_q_len=shp.max_q_len)


# A mixer's ``run`` writes the columns that the output projection ``out_weight`` [width, columns] reads; a feed-forward likewise.
class AttentionMixer:
    """Grouped-query attention: one product for q, k, v and the gate, short convolution + norms + rotation + value mixing + cache write in
    one kernel, attention with sink and gate in its epilogue."""

    def __init__(self, s: AttentionSpec, pk: _Packer):
        self.s, self.rot = s, _Rotation(s.rotary, pk.device)
        self.dk, self.dv = _up(s.dim, 16), _up(s.vdim, 16)
        pads = {"q": (s.heads, self.dk), "k": (s.kv_heads, self.dk), "v": (s.kv_heads, self.dv)}
        parts = [_pad_rows(pk.raw("mix", key), *pad) for key, pad in pads.items()]
        if s.head_gate:
            parts.append(pk.raw("mix", "g"))
        elif s.gated:
            parts.append(_pad_rows(pk.raw("mix", "g"), s.heads, self.dv))
        self.k_off = s.heads * self.dk
        self.v_off = self.k_off + s.kv_heads * self.dk
        self.g_off = self.v_off + s.kv_heads * self.dv
        self.proj = pk.linear(torch.cat(parts, 0))
        self.out_weight = _pad_cols(pk.raw("mix", "o"), s.heads, self.dv)
        self.q_norm = pk.f32("mix", "q.norm") if s.qk_norm else None
        self.k_norm = pk.f32("mix", "k.norm") if s.qk_norm else None
        self.sink = pk.f32("mix", "sink") if s.sink else None
        self.conv = _ShortConv([_pad_rows(pk.raw("mix", key + ".conv"), *pad) for key, pad in pads.items()]) if s.taps else None
        self.v_mode, self.v_mix = 0, 0.0           # set by the executor's weights: 1 = first layer that mixes values, 2 = a later one
        if s.v_mix:
            self.v_mode, self.v_mix = 2, float(pk.raw("mix", "vmix").float())

    def allocate(self, ex: "LayeredExecutor") -> None:
        shape = (ex.num_kv_blocks, self.s.kv_heads, ex.block_size)
        self.k_cache = torch.zeros(shape + (self.dk,), dtype=ex.dtype, device=ex.device)
        self.v_cache = torch.zeros(shape + (self.dv,), dtype=ex.dtype, device=ex.device)
        if self.conv:
            self.conv.allocate(ex)

    def state(self) -> List[torch.Tensor]:
        return [self.conv.ring] if self.conv else []

    def cache_bytes(self) -> int:
        return self.k_cache.nbytes + self.v_cache.nbytes + sum(t.nbytes for t in self.state())

    def run(self, ex: "LayeredExecutor", sb: "LayeredStepBuffers", shp: StepShape, x: torch.Tensor, out: torch.Tensor) -> None:
        s, T = self.s, shp.T
        proj = sb.scratch("proj", T, self.proj.N)
        K.gemm(x, self.proj, out=proj, ws=ex.ws)
        q, extra = proj, {}
        if self.conv:
            q = sb.scratch("queries", T, self.k_off)
            extra.update(self.conv.args(sb, shp), q_out=q, ldq=q.stride(0))
        if self.v_mode:
            first = sb.scratch("v_first", T, s.kv_heads * s.vdim)
            extra.update(v_first=first, ld_vf=first.stride(0), v_mode=self.v_mode, v_mix=self.v_mix)
        if self.rot.dims:
            extra.update(rot_dims=self.rot.dims, rope=ex.rope(sb, shp, self.rot))
        K.heads_prepare(proj=proj, k_cache=self.k_cache, v_cache=self.v_cache, q_norm=self.q_norm, k_norm=self.k_norm, positions=sb.view("positions"),
                        slot_map=sb.view("slot_map"), T=T, H=s.heads, G=s.kv_heads, D=s.dim, Dv=s.vdim, dk_pad=self.dk, dv_pad=self.dv, ldp=proj.stride(0),
                        k_off=self.k_off, v_off=self.v_off, block_size=ex.block_size, dtype=ex.storage, eps=ex.cfg.norm_eps, **extra)
        gate = {}
        if s.gated or s.head_gate:
            gate = dict(gate=proj[:, self.g_off:], ld_gate=proj.stride(0), gate_head=1 if s.head_gate else self.dv, gate_scalar=int(s.head_gate))
        ex.attention(sb, shp, q=q, k=self.k_cache, v=self.v_cache, out=out, Hq=s.heads, Hkv=s.kv_heads, Dk=self.dk, Dv=s.vdim, ldq=q.stride(0),
                     q_head=self.dk, k_row=self.dk, v_row=self.dv, ldo=out.stride(0), o_head=self.dv, window=s.window, chunk=s.chunk, sink=self.sink,
                     scale=s.scale, **gate)
        ex.kernel_launches += 3 + (self.conv is not None and shp.max_q_len > 1 and self.conv.taps > 1)


class LatentAttentionMixer:
    """Latent attention over the cached low-rank rows, in one of two forms of the same sums. Absorbed: the key projection moves to the
    query (q W_uk) and the value projection behind the weighted sum, so that all heads attend to the one cached row per token; the
    form of decoding, of fp32 and of head sizes that the prefill kernel does not serve. Expanded: the rows that the step's windows
    reach become per-head keys and values; fewer operations when many new tokens share them (prefill)."""

    def __init__(self, s: LatentAttentionSpec, pk: _Packer):
        self.s, self.rot = s, _Rotation(s.rotary, pk.device)
        H, D, R, C, Dv = s.heads, s.dim, s.rot_dim, s.kv_rank, s.vdim
        self.dp, self.rp, self.cp, self.dv = _up(D, 16), _up(R, 16), _up(C, 16), _up(Dv, 16)
        self.q_pitch, self.row = self.dp + self.rp, self.cp + self.rp
        self.pitch = self.row + 8         # a cached row: an odd number of 16-byte pieces, so that pages copied to shared memory as they are read without bank conflicts
        q = pk.raw("mix", "q").reshape(H, D + R, -1)
        q = torch.cat([_pad_rows(q[:, :D].reshape(H * D, -1), H, self.dp).reshape(H, self.dp, -1),
                       _pad_rows(q[:, D:].reshape(H * R, -1), H, self.rp).reshape(H, self.rp, -1)], 1).reshape(H * self.q_pitch, -1)
        dkv = pk.raw("mix", "dkv")
        self.c_off = H * self.q_pitch
        self.kr_off = self.c_off + self.cp
        self.proj = pk.linear(torch.cat([q, _pad_rows(dkv[:C], 1, self.cp), _pad_rows(dkv[C:], 1, self.rp)], 0))
        self.c_norm = pk.f32("mix", "dkv.norm")
        self.uk = pk.block_diag(pk.raw("mix", "uk").reshape(H, D, C).transpose(1, 2))
        self.uv = pk.block_diag(pk.raw("mix", "uv").reshape(H, Dv, C))
        self.out_weight = _pad_cols(pk.raw("mix", "o"), H, self.dv)
        self.k_head, self.v_head = _up(D, 64), _up(Dv, 64)
        self.ukv = None
        if pk.dtype == torch.bfloat16 and self.k_head <= 128 and R <= 64 and self.v_head <= 128 and s.scale > 0:
            self.ukv = pk.linear(torch.cat([_pad_rows(pk.raw("mix", "uk"), H, self.k_head), _pad_rows(pk.raw("mix", "uv"), H, self.v_head)], 0))

    def _expanded_rows(self, sb: "LayeredStepBuffers", shp: StepShape) -> int:
        """Cached rows that this step's windows reach (as csrc/cuda/attention.cuh counts them), or 0: run the absorbed form."""
        if self.ukv is None or shp.spans is None:
            return 0
        first = lambda past: max(0, past - self.s.window + 1) // 128 * 128 if self.s.window > 0 else 0
        rows = sum(past + new - first(past) for past, new in shp.spans)
        return rows if rows <= 2 * sb.Tcap else 0

    def allocate(self, ex: "LayeredExecutor") -> None:
        self.cache = torch.zeros((ex.num_kv_blocks, ex.block_size, self.pitch), dtype=ex.dtype, device=ex.device)

    def state(self) -> List[torch.Tensor]:
        return []

    def cache_bytes(self) -> int:
        return self.cache.nbytes

    def run(self, ex: "LayeredExecutor", sb: "LayeredStepBuffers", shp: StepShape, x: torch.Tensor, out: torch.Tensor) -> None:
        s, T, H = self.s, shp.T, self.s.heads
        proj = sb.scratch("proj", T, self.proj.N)
        K.gemm(x, self.proj, out=proj, ws=ex.ws)
        rows = self._expanded_rows(sb, shp)
        q = proj if rows else sb.scratch("latent_q", T, H * self.row)
        q_rot = dict(q_rot=proj[:, self.dp:], ld_qr=proj.stride(0), qr_pitch=self.q_pitch) if rows else \
            dict(q_rot=q[:, self.cp:], ld_qr=q.stride(0), qr_pitch=self.row)
        K.latent_prepare(proj=proj, cache=self.cache, c_norm=self.c_norm, positions=sb.view("positions"), slot_map=sb.view("slot_map"), T=T,
                         H=H, C=s.kv_rank, R=s.rot_dim, q_pitch=self.q_pitch, q_rot_off=self.dp, c_off=self.c_off, kr_off=self.kr_off, ldp=proj.stride(0),
                         row_pitch=self.pitch, key_off=self.cp, block_size=ex.block_size, dtype=ex.storage, eps=ex.cfg.norm_eps, **q_rot, **self.rot.args())
        if rows:
            self._attend_expanded(ex, sb, shp, rows, proj, out)
        else:
            self._attend_absorbed(ex, sb, shp, proj, q, out)
        ex.kernel_launches += 2

    def _attend_expanded(self, ex, sb, shp: StepShape, rows: int, proj: torch.Tensor, attn: torch.Tensor) -> None:
        s, H = self.s, self.s.heads
        batch = dict(past_lens=sb.view("past_lens"), subsequence_begins=sb.view("subsequence_begins"), block_indices=sb.view("block_indices"),
                     block_indices_begins=sb.view("block_indices_begins"), B=shp.B, window=s.window, block_size=ex.block_size)
        lat = sb.scratch("latent_rows", rows, self.ukv.K, cap=2 * sb.Tcap)
        kv = sb.scratch("latent_kv", rows, self.ukv.N, cap=2 * sb.Tcap)
        K.latent_gather(cache=self.cache, out=lat, kv_rows=sb.kv_rows, rows=rows, cols=self.cp, row_pitch=self.pitch, out_pitch=lat.stride(0), **batch)
        K.gemm(lat, self.ukv, out=kv, ws=ex.ws)
        K.latent_prefill(q=proj, kv=kv, cache=self.cache, out=attn, kv_rows=sb.kv_rows, T=shp.T, H=H, rows=rows, R=s.rot_dim, Dv=self.dv, ldq=proj.stride(0),
                         q_head=self.q_pitch, q_rot_off=self.dp, ld_kv=kv.stride(0), k_head=self.k_head, v_off=H * self.k_head, v_head=self.v_head,
                         row_pitch=self.pitch, key_off=self.cp, ldo=attn.stride(0), o_head=self.dv, scale=s.scale, **batch)
        ex.kernel_launches += 3

    def _attend_absorbed(self, ex, sb, shp: StepShape, proj: torch.Tensor, q: torch.Tensor, attn: torch.Tensor) -> None:
        s, T, H = self.s, shp.T, self.s.heads
        K.gemm_block_diag(proj[:, :self.c_off], self.uk, q, self.q_pitch, self.row, ws=ex.ws)
        lat = sb.scratch("latent_o", T, H * self.cp)
        ex.attention(sb, shp, q=q, k=self.cache, v=self.cache, out=lat, Hq=H, Hkv=1, Dk=self.row, Dv=s.kv_rank, ldq=q.stride(0), q_head=self.row,
                     k_row=self.pitch, v_row=self.pitch, ldo=lat.stride(0), o_head=self.cp, window=s.window, scale=s.scale)
        K.gemm_block_diag(lat[:, :H * self.cp], self.uv, attn, self.cp, self.dv, ws=ex.ws)
        ex.kernel_launches += 3


class RgLruMixer:
    """Griffin's recurrent block: one product for both branches, convolution, block-diagonal gate product, recurrence with the
    other branch's activation in its epilogue, output projection. State per request slot, fp32."""

    def __init__(self, s: RgLruSpec, pk: _Packer):
        self.s = s
        N, B = s.width, s.blocks
        if N % B:
            raise ValueError("recurrent width %d is not a multiple of its %d blocks" % (N, B))
        self.bw = N // B
        self.bp, self.np = _up(self.bw, 16), _up(N, 8)
        pad = lambda t: torch.nn.functional.pad(t, (0, self.np - N))
        self.proj = pk.linear(torch.cat([_pad_rows(pk.raw("mix", "y"), 1, self.np), _pad_rows(pk.raw("mix", "x"), 1, self.np)], 0),
                              torch.cat([pad(pk.raw("mix", "y.b")), pad(pk.raw("mix", "x.b"))]))
        self.out_weight = pk.raw("mix", "o")
        self.conv_w = pk.raw("mix", "conv").float().t().contiguous()          # [taps, N]
        self.conv_b = pk.f32("mix", "conv.b")
        ra, ri = pk.raw("mix", "ra"), pk.raw("mix", "ri")
        grow = lambda w: torch.nn.functional.pad(w, (0, 0, 0, self.bp - self.bw))
        self.gates = pk.block_diag(torch.cat([grow(ra), grow(ri)], 1))        # [B, 2 * bp, bw]
        self.gate_b = torch.stack([pk.f32("mix", "ra.b"), pk.f32("mix", "ri.b")]).contiguous()
        self.log_decay = (s.decay * torch.nn.functional.softplus(pk.raw("mix", "lam").double())).float().contiguous()

    def allocate(self, ex: "LayeredExecutor") -> None:
        self.lru_state = torch.zeros((ex.num_slots, self.s.width), dtype=torch.float32, device=ex.device)
        self.conv_state = torch.zeros((ex.num_slots, max(self.s.taps - 1, 1), self.s.width), dtype=torch.float32, device=ex.device)

    def state(self) -> List[torch.Tensor]:
        return [self.lru_state, self.conv_state]

    def cache_bytes(self) -> int:
        return self.lru_state.nbytes + self.conv_state.nbytes

    def run(self, ex: "LayeredExecutor", sb: "LayeredStepBuffers", shp: StepShape, x: torch.Tensor, out: torch.Tensor) -> None:
        s, T = self.s, shp.T
        proj = sb.scratch("proj", T, self.proj.N)
        K.gemm(x, self.proj, out=proj, ws=ex.ws)
        u = sb.scratch("lru_u", T, s.blocks * self.bp)
        gates = sb.scratch("lru_gates", T, s.blocks * 2 * self.bp, torch.float32)
        args = dict(x=proj[:, self.np:], y=proj, u=u, out=out, gates=gates, gate_b=self.gate_b, log_decay=self.log_decay, conv_w=self.conv_w,
                    conv_b=self.conv_b, state=self.lru_state, conv_state=self.conv_state, subsequence_begins=sb.view("subsequence_begins"),
                    past_lens=sb.view("past_lens"), slots=sb.view("state_slots"), B=shp.B, T=T, N=s.width, taps=s.taps, bw=self.bw, ub_pitch=self.bp,
                    gb_pitch=2 * self.bp, gi_off=self.bp, ldx=proj.stride(0), ldy=proj.stride(0), ldu=u.stride(0), ldg=gates.stride(0), ldo=out.stride(0),
                    max_q_len=shp.max_q_len, dtype=ex.storage)
        K.causal_conv(**args)
        K.gemm_block_diag(u, self.gates, gates, self.bp, 2 * self.bp, ws=ex.ws)
        K.lru_scan(**args)
        ex.kernel_launches += 4


class ChannelDeltaMixer:
    """Gated delta rule with a decay per key channel: one product for q, k, v, step sizes and the inner halves of the two low-rank
    projections, one block-diagonal product for their outer halves (fp32), one kernel for everything else."""

    def __init__(self, s: ChannelDeltaSpec, pk: _Packer):
        self.s = s
        self.dk, self.dv = _up(s.dim, 16), _up(s.vdim, 16)
        H, G = s.heads, s.kv_heads
        pads = {"q": (G, self.dk), "k": (G, self.dk), "v": (H, self.dv)}
        self.k_off = G * self.dk
        self.v_off = 2 * self.k_off
        self.b_off = self.v_off + H * self.dv
        self.low_off = self.b_off + _up(H, 16)
        a1, a2, g1, g2 = (pk.raw("mix", key) for key in ("a1", "a2", "g1", "g2"))
        if a1.shape[0] != a2.shape[1] or g1.shape[0] != g2.shape[1]:
            raise ValueError("layer %d: the halves of a low-rank projection do not fit each other" % pk.layer)
        self.rank = _up(max(a1.shape[0], g1.shape[0]), 16)                         # columns of an inner half
        self.proj = pk.linear(torch.cat([_pad_rows(pk.raw("mix", key), *pad) for key, pad in pads.items()] + [
            _pad_rows(pk.raw("mix", "b"), 1, _up(H, 16)), _pad_rows(a1, 1, self.rank), _pad_rows(g1, 1, self.rank)], 0))
        a2, g2 = _pad_rows(a2, H, self.dk), _pad_rows(g2, H, self.dv)
        self.low_n = max(a2.shape[0], g2.shape[0])
        grow = lambda w: torch.nn.functional.pad(w, (0, self.rank - w.shape[1], 0, self.low_n - w.shape[0]))
        self.low = pk.block_diag(torch.stack([grow(a2), grow(g2)]))               # [2, low_n, rank]
        self.out_weight = _pad_cols(pk.raw("mix", "o"), H, self.dv)
        self.conv = _ShortConv([_pad_rows(pk.raw("mix", key + ".conv"), *pad) for key, pad in pads.items()])
        self.decay_a = pk.raw("mix", "A_log").float().exp().contiguous()
        self.dt_bias = torch.nn.functional.pad(pk.raw("mix", "dt_bias").float().reshape(H, s.dim), (0, self.dk - s.dim)).contiguous()
        self.norm = pk.f32("mix", "norm", 16)

    def allocate(self, ex: "LayeredExecutor") -> None:
        self.delta_state = torch.zeros((ex.num_slots, self.s.heads, self.dk, self.dv), dtype=torch.float32, device=ex.device)
        self.conv.allocate(ex)

    def state(self) -> List[torch.Tensor]:
        return [self.delta_state, self.conv.ring]

    def cache_bytes(self) -> int:
        return sum(t.nbytes for t in self.state())

    def run(self, ex: "LayeredExecutor", sb: "LayeredStepBuffers", shp: StepShape, x: torch.Tensor, out: torch.Tensor) -> None:
        s, T = self.s, shp.T
        proj = sb.scratch("proj", T, self.proj.N)
        K.gemm(x, self.proj, out=proj, ws=ex.ws)
        low = sb.scratch("delta_low", T, 2 * self.low_n, torch.float32)
        K.gemm_block_diag(proj[:, self.low_off:], self.low, low, self.rank, self.low_n, ws=ex.ws)
        # (what the kernel prepares for all groups of tokens at once; the largest step decides the size)
        records = sb.scratch("delta_records", 1, K.channel_delta_record_floats(sb.Tcap, sb.Bcap, s.heads, self.dk, self.dv), torch.float32, cap=1)
        K.channel_delta(proj=proj, low=low, records=records, decay_a=self.decay_a, dt_bias=self.dt_bias, norm=self.norm, state=self.delta_state, out=out, T=T, H=s.heads,
                        G=s.kv_heads, D=s.dim, Dv=s.vdim, dk=self.dk, dv=self.dv, ldp=proj.stride(0), k_off=self.k_off, v_off=self.v_off, b_off=self.b_off,
                        ld_low=low.stride(0), gate_off=self.low_n, ldo=out.stride(0), o_head=self.dv, dtype=ex.storage, q_scale=s.dim ** -0.5,
                        eps=ex.cfg.norm_eps, **self.conv.args(sb, shp))
        ex.kernel_launches += 3 + (shp.max_q_len > 1 and self.conv.taps > 1)


class LimitedGlu:
    """Gated MLP with clamped halves; in bf16 the activation runs in the epilogue of the gate / up product."""

    def __init__(self, s: LimitedGluSpec, pk: _Packer):
        self.s, self.fp = s, _up(s.ff, 64)
        gate, up = _pad_rows(pk.raw("mlp", "gate"), 1, self.fp), _pad_rows(pk.raw("mlp", "up"), 1, self.fp)
        self.fused = pk.dtype == torch.bfloat16
        self.gate_up = pk.linear(K.interleave_gate_up(gate, up) if self.fused else torch.cat([gate, up], 0))
        self.out_weight = pk.raw("mlp", "down")

    def run(self, ex: "LayeredExecutor", sb: "LayeredStepBuffers", shp: StepShape, x: torch.Tensor, act: torch.Tensor) -> None:
        s = self.s
        if self.fused:
            K.gemm(x, self.gate_up, out=act, act=K.ACT_GLU_LIMITED, glu=(s.limit, s.slope, s.shift), ws=ex.ws)
        else:
            gu = sb.scratch("mlp_gu", shp.T, 2 * self.fp)
            K.gemm(x, self.gate_up, out=gu, ws=ex.ws)
            K.glu_limited(gu, act, s.ff, self.fp, s.limit, s.slope, s.shift)
            ex.kernel_launches += 1
        ex.kernel_launches += 1


class SquaredRelu:
    """MLP with relu(up)^2; the activation runs in the epilogue of the up product."""

    def __init__(self, s: SquaredReluSpec, pk: _Packer):
        self.fp = _up(s.ff, 64)
        self.up = pk.linear(_pad_rows(pk.raw("mlp", "up"), 1, self.fp))
        self.out_weight = pk.raw("mlp", "down")

    def run(self, ex: "LayeredExecutor", sb: "LayeredStepBuffers", shp: StepShape, x: torch.Tensor, act: torch.Tensor) -> None:
        K.gemm(x, self.up, out=act, act=K.ACT_RELU2, ws=ex.ws)
        ex.kernel_launches += 1


MIXERS = {AttentionSpec: AttentionMixer, LatentAttentionSpec: LatentAttentionMixer, RgLruSpec: RgLruMixer, ChannelDeltaSpec: ChannelDeltaMixer}
MLPS = {LimitedGluSpec: LimitedGlu, SquaredReluSpec: SquaredRelu}


class _Layer:
    """``out``: one output product over [mixer columns | feed-forward columns] of a parallel layer, else the mixer's (``down``: the
    feed-forward's). ``mix_cols`` / ``mlp_cols``: columns that mixer and feed-forward write, whole k-blocks of the product."""

    def __init__(self, spec, pk: _Packer, parallel: bool):
        self.mixer = MIXERS[type(spec.mixer)](spec.mixer, pk)
        self.mlp = MLPS[type(spec.mlp)](spec.mlp, pk) if spec.mlp is not None else None
        self.norm1 = pk.f32("norm", "1", 4)
        self.norm2 = pk.f32("norm", "2", 4) if spec.mlp is not None else None
        subs = [self.mixer] + ([self.mlp] if self.mlp is not None else [])
        widths = [_up(sub.out_weight.shape[1], 64) for sub in subs]
        weights = [torch.nn.functional.pad(sub.out_weight, (0, n - sub.out_weight.shape[1])) for sub, n in zip(subs, widths)]
        for sub in subs:
            sub.out_weight = None
        self.mix_cols, self.mlp_cols = widths[0], sum(widths[1:])
        self.out = pk.linear(torch.cat(weights, 1) if parallel else weights[0])
        self.down = pk.linear(weights[1]) if self.mlp is not None and not parallel else None


class LayeredWeights:
    """All weights of a layered decoder on the device, in kernel layout."""

    def __init__(self, ckpt: Checkpoint, device, dtype: torch.dtype = torch.bfloat16):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("layered decoders are served in bfloat16 or float32")
        cfg = self.config = ckpt.config
        self.dtype = dtype
        self.layers = [_Layer(spec, _Packer(ckpt, i, device, dtype), cfg.block == PARALLEL_NORM) for i, spec in enumerate(cfg.layers)]
        mixing = [layer.mixer for layer in self.layers if getattr(layer.mixer, "v_mode", 0)]
        if any(m.s.kv_heads * m.s.vdim != mixing[0].s.kv_heads * mixing[0].s.vdim for m in mixing):
            raise ValueError("layers that mix values must have the same number of value columns")
        for m in mixing[:1]:
            m.v_mode = 1
        pk = _Packer(ckpt, -1, device, dtype)
        self.embed = pk.raw("", "embed").to(dtype).contiguous()
        self.embed_norm = pk.f32("", "embed.norm", 4) if cfg.embed_norm else None
        self.final_norm = pk.f32("", "final.norm", 4)
        self.head = pk.linear(pk.raw("", "head"))


class LayeredStepBuffers(StepBuffers):
    """Descriptor, fp32 residual stream ``h``, what the products of a layer read in the compute type (``x``: its copy, or ``h`` itself in
    fp32; ``x`` and ``x2``: its two norms in parallel layers), sublayer output ``y`` and named scratch that layers share."""

    def __init__(self, cfg: LayeredConfig, dtype: torch.dtype, Tcap: int, Bcap: int, max_blocks_per_seq: int, device):
        super().__init__(Tcap, Bcap, max_blocks_per_seq, device, cfg.vocab_size, logits_dtype=torch.float32, state_slots=True)
        width = _up(cfg.hidden_size, 64)
        zeros = lambda rows, dt: torch.zeros((rows, width), dtype=dt, device=device)
        self.h, self.y = zeros(Tcap, torch.float32), zeros(Tcap, torch.float32)
        parallel = cfg.block == PARALLEL_NORM
        self.x = self.h if dtype == torch.float32 and not parallel else zeros(Tcap, dtype)
        self.x2 = zeros(Tcap, dtype) if parallel else None
        self.ropes: Dict[tuple, torch.Tensor] = {}      # angle tables of the step, by rotation
        self.last_x = zeros(Bcap, dtype)
        self.kv_rows = torch.zeros(Bcap + 1, dtype=torch.int32, device=device)
        self.device, self.dtype = device, dtype
        self._scratch: Dict[tuple, torch.Tensor] = {}

    def scratch(self, name: str, rows: int, cols: int, dtype: Optional[torch.dtype] = None, cap: int = 0) -> torch.Tensor:
        """[rows, cols] view of a buffer of ``cap`` (default: Tcap) rows that starts out as zeros; its row pitch is a multiple of 64."""
        dtype = dtype or self.dtype
        key = (name, cols, dtype)
        if key not in self._scratch:
            self._scratch[key] = torch.zeros((cap or self.Tcap, _up(cols, 64)), dtype=dtype, device=self.device)
        return self._scratch[key][:rows, :cols]


class LayeredExecutor(LlmExecutor):
    """Runs steps of a layered decoder on one GPU."""

    def __init__(self, weights: LayeredWeights, num_kv_blocks: int, block_size: int = 16, max_batch_tokens: int = 8192, max_seqs: int = 64,
                 max_blocks_per_seq: int = 0, device="cuda", use_cuda_graphs: bool = True):
        cfg = weights.config
        super().__init__(cfg, num_kv_blocks, block_size, max_seqs, max_blocks_per_seq, device, use_cuda_graphs)
        self.w, self.dtype, self.storage = weights, weights.dtype, K.storage_type(weights.dtype)
        self.has_recurrent_state = cfg.has_recurrent_state
        for layer in weights.layers:
            layer.mixer.allocate(self)
        make = lambda Tcap: LayeredStepBuffers(cfg, self.dtype, Tcap, max_seqs, self.max_blocks_per_seq, self.device)
        self.prefill, self.decode = make(max_batch_tokens), make(max_seqs)

    def _recurrent_state(self) -> List[torch.Tensor]:
        return [t for layer in self.w.layers for t in layer.mixer.state()]

    def kv_cache_bytes(self) -> int:
        return sum(layer.mixer.cache_bytes() for layer in self.w.layers)

    def attention(self, sb: LayeredStepBuffers, shp: StepShape, **kw) -> None:
        """Paged attention of this step's tokens (``K.window_attention``) with the batch description filled in."""
        K.window_attention(past_lens=sb.view("past_lens"), subsequence_begins=sb.view("subsequence_begins"), block_indices=sb.view("block_indices"),
                           block_indices_begins=sb.view("block_indices_begins"), B=shp.B, T=shp.T, block_size=self.block_size,
                           max_context_len=shp.max_ctx, max_q_len=shp.max_q_len, dtype=self.storage, scratch=self.ws.pa_scratch,
                           scratch_bytes=self.ws.pa_scratch.nbytes, exact=1 if self.dtype == torch.float32 else 0, **kw)

    def rope(self, sb: LayeredStepBuffers, shp: StepShape, rot: _Rotation) -> torch.Tensor:
        """(cos, sin) of the step's positions for a rotation; computed by the first layer that asks for it."""
        key = (rot.dims, rot.mult, rot.freq)
        if key not in sb.ropes:
            table = sb.scratch("rope %s" % (key,), shp.T, rot.dims, torch.float32)
            table = table.as_strided((shp.T, rot.dims), (rot.dims, 1))            # no gaps between tokens
            K.rope_table(sb.view("positions"), rot.inv_freq, table, rot.mult)
            self.kernel_launches += 1
            sb.ropes[key] = table
        return sb.ropes[key]

    def _norm(self, sb: LayeredStepBuffers, T: int, w: torch.Tensor) -> None:
        """x <- norm(residual_scale * x + y), in fp32, plus the copy that the next products read."""
        cfg = self.cfg
        K.sum_rmsnorm(sb.h[:T], w, cfg.norm_eps, cfg.hidden_size, y=sb.y[:T], alpha=cfg.residual_scale, w_offset=cfg.norm_offset, h_out=sb.h[:T],
                      x_out=None if sb.x is sb.h else sb.x[:T])

    def _forward(self, sb: LayeredStepBuffers, shp: StepShape) -> None:
        T, B = shp.T, shp.B
        ids = sb.view("ids")[:T]
        K.resolve_ids(ids, sb.view("tok_src")[:T], self.last_token)
        copy = None if sb.x is sb.h or self.cfg.block == PARALLEL_NORM else sb.x       # (parallel layers start with their norms)
        K.stream_embed(ids, self.w.embed, sb.h, copy)
        sb.ropes.clear()
        if self.w.embed_norm is not None:
            K.sum_rmsnorm(sb.h[:T], self.w.embed_norm, self.cfg.norm_eps, self.cfg.hidden_size, w_offset=self.cfg.norm_offset, h_out=sb.h[:T],
                          x_out=None if copy is None else copy[:T])
            self.kernel_launches += 1
        if self.cfg.block == PARALLEL_NORM:
            self._parallel_layers(sb, shp)
        else:
            self._post_norm_layers(sb, shp)
        self._logits(sb, sb.view("logit_idx")[:B], sb.logits[:B])
        self.kernel_launches += 2 + 3
        self._sample(sb, B)

    def _post_norm_layers(self, sb: LayeredStepBuffers, shp: StepShape) -> None:
        T = shp.T
        x, y = sb.x[:T], sb.y[:T]
        for layer in self.w.layers:
            heads = sb.scratch("heads", T, layer.mix_cols)
            layer.mixer.run(self, sb, shp, x, heads)
            K.gemm(heads, layer.out, out=y, out_f32=True, ws=self.ws)
            self._norm(sb, T, layer.norm1)
            self.kernel_launches += 2
            if layer.mlp is not None:
                act = sb.scratch("mlp_act", T, layer.mlp_cols)
                layer.mlp.run(self, sb, shp, x, act)
                K.gemm(act, layer.down, out=y, out_f32=True, ws=self.ws)
                self._norm(sb, T, layer.norm2)
                self.kernel_launches += 2

    def _parallel_layers(self, sb: LayeredStepBuffers, shp: StepShape) -> None:
        """The output of a layer stays in ``y`` until the next layer's norms (or the final one) add it to the stream."""
        cfg, T = self.cfg, shp.T
        h, x, x2, y = sb.h[:T], sb.x[:T], sb.x2[:T], sb.y[:T]
        for i, layer in enumerate(self.w.layers):
            second = dict(w2=layer.norm2, x2_out=x2) if layer.mlp is not None else {}
            K.sum_rmsnorm(h, layer.norm1, cfg.norm_eps, cfg.hidden_size, y=y if i else None, w_offset=cfg.norm_offset, s_out=h if i else None, x_out=x, **second)
            both = sb.scratch("heads", T, layer.mix_cols + layer.mlp_cols)
            layer.mixer.run(self, sb, shp, x, both[:, :layer.mix_cols])
            if layer.mlp is not None:
                layer.mlp.run(self, sb, shp, x2, both[:, layer.mix_cols:])
            K.gemm(both, layer.out, out=y, out_f32=True, ws=self.ws)
            self.kernel_launches += 2

    def _logits(self, sb: LayeredStepBuffers, rows: torch.Tensor, out: torch.Tensor) -> None:
        cfg, x = self.cfg, sb.last_x[:rows.shape[0]]
        y = sb.y if cfg.block == PARALLEL_NORM and self.w.layers else None
        K.sum_rmsnorm(sb.h, self.w.final_norm, cfg.norm_eps, cfg.hidden_size, y=y, w_offset=cfg.norm_offset, x_out=x, row_idx=rows)
        K.gemm(x, self.w.head, out=out, out_f32=True, act=K.ACT_SOFTCAP if cfg.logit_softcap > 0 else K.ACT_NONE, cap=cfg.logit_softcap, ws=self.ws)

    def logits_at(self, sb: LayeredStepBuffers, rows: List[int]) -> torch.Tensor:
        """Logits (fp32) after the step that ``sb`` holds, at the given token rows of its batch."""
        idx = torch.tensor(rows, dtype=torch.int32, device=self.device)
        out = torch.empty((len(rows), self.cfg.vocab_size), dtype=torch.float32, device=self.device)
        for i in range(0, len(rows), sb.Bcap):
            self._logits(sb, idx[i:i + sb.Bcap], out[i:i + sb.Bcap])
        return out


def create_executor(ckpt: Checkpoint, device_index: int = 0, max_num_seqs: int = 64, max_num_batched_tokens: int = 8192, max_model_len: int = 4096,
                    block_size: int = 16, kv_cache_blocks: int = 0, properties: Optional[dict] = None):
    """Executor of a checkpoint and the scheduler limits that fit it: ``(executor, SchedulerConfig)``. ``properties``:
    INFERENCE_PRECISION_HINT (bf16 / f32), CUDA_USE_GRAPHS, dynamic_split_fuse; others are refused."""
    from .. import properties as props
    from ..genai.scheduler import SchedulerConfig
    opts = {str(k): v for k, v in (properties or {}).items()}
    precision = str(opts.pop(str(props.hint.inference_precision), "bf16")).lower()
    dtypes = {"bf16": torch.bfloat16, "bfloat16": torch.bfloat16, "f32": torch.float32, "float32": torch.float32}
    if precision not in dtypes:
        raise ValueError("a checkpoint is served in bf16 or f32, not '%s'" % precision)
    graphs = str(opts.pop(str(props.cuda.use_cuda_graphs), True)).upper() not in ("FALSE", "NO", "0")
    fuse = bool(opts.pop("dynamic_split_fuse", False))
    if opts:
        raise ValueError("unknown properties for a checkpoint: %s" % ", ".join(sorted(opts)))
    device = torch.device("cuda", device_index)
    blocks_per_seq = (max_model_len + block_size - 1) // block_size + 1
    num_blocks = kv_cache_blocks or max_num_seqs * blocks_per_seq + 8
    with torch.cuda.device(device), torch.no_grad():
        ex = LayeredExecutor(LayeredWeights(ckpt, device, dtypes[precision]), num_kv_blocks=num_blocks, block_size=block_size,
                             max_batch_tokens=max_num_batched_tokens, max_seqs=max_num_seqs, max_blocks_per_seq=blocks_per_seq, device=device,
                             use_cuda_graphs=graphs)
    return ex, SchedulerConfig(max_num_batched_tokens=max_num_batched_tokens, max_num_seqs=max_num_seqs, num_kv_blocks=num_blocks, block_size=block_size,
                               max_blocks_per_seq=blocks_per_seq, dynamic_split_fuse=fuse)

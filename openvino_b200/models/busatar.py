"""Busatar: its ``config.json`` and the names of its tensors, in terms of the layered decoder (``LayeredConfig``).

Three token mixers (latent attention, grouped-query attention with normed heads and a gated output, Griffin's recurrent block),
an optional clamped gated MLP per layer, and a norm after every residual sum with weights stored around zero.
"""
from __future__ import annotations

from .llm_config import AttentionSpec, LatentAttentionSpec, LayeredConfig, LayerSpec, LimitedGluSpec, RgLruSpec, RotarySpec


def _rotary(rot: dict) -> RotarySpec:
    s = rot.get("scaling")
    yarn = (float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None
    return RotarySpec(int(rot["dims"]), float(rot["base"]), yarn)


def _window(m: dict) -> int:
    return int(m["mask"]["size"])


def _mixer(kind: str, m: dict):
    if kind == "attention":
        return AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), _window(m), qk_norm=True, gated=True)
    if kind == "latent_attention":
        return LatentAttentionSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]), _rotary(m["rot"]),
                                   _window(m))
    if kind == "rglru":
        return RgLruSpec(int(m["width"]), int(m["blocks"]), int(m["conv"]))
    raise ValueError("unknown token mixer '%s'" % kind)


def _mlp(m):
    if m is None:
        return None
    if m["kind"] != "dense":
        raise ValueError("unknown feed-forward '%s'" % m["kind"])
    return LimitedGluSpec(int(m["ff"]), float(m["limit"]))


def read_config(cfg: dict) -> LayeredConfig:
    layers = tuple(LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in cfg["layers"])
    return LayeredConfig("Busatar", int(cfg["vocab"]), int(cfg["width"]), layers, norm_eps=float(cfg["norm"]["eps"]),
                         residual_scale=float(cfg["postln_alpha"]), norm_offset=1.0)


def tensor_name(layer: int, part: str, key: str) -> str:
    """Name in the checkpoint. ``part``: "mix" / "mlp" / "norm" (key "1" or "2") of a layer; layer -1: "embed", "final.norm", "head"."""
    if layer < 0:
        return key
    return "l%d.norm%s" % (layer, key) if part == "norm" else "l%d.%s.%s" % (layer, part, key)


def tensor_shapes(cfg: LayeredConfig) -> dict:
    """Name -> shape of every tensor of a checkpoint."""
    W = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, W), "final.norm": (W,), "head": (cfg.vocab_size, W)}
    for i, layer in enumerate(cfg.layers):
        m, mix = layer.mixer, {}
        if isinstance(m, AttentionSpec):
            mix = {"q": (m.heads * m.dim, W), "k": (m.kv_heads * m.dim, W), "v": (m.kv_heads * m.vdim, W), "q.norm": (m.dim,), "k.norm": (m.dim,),
                   "g": (m.heads * m.vdim, W), "o": (W, m.heads * m.vdim)}
        elif isinstance(m, LatentAttentionSpec):
            mix = {"q": (m.heads * (m.dim + m.rot_dim), W), "dkv": (m.kv_rank + m.rot_dim, W), "dkv.norm": (m.kv_rank,), "uk": (m.heads * m.dim, m.kv_rank),
                   "uv": (m.heads * m.vdim, m.kv_rank), "o": (W, m.heads * m.vdim)}
        elif isinstance(m, RgLruSpec):
            N, B = m.width, m.blocks
            mix = {"y": (N, W), "y.b": (N,), "x": (N, W), "x.b": (N,), "conv": (N, m.taps), "conv.b": (N,), "ra": (B, N // B, N // B), "ra.b": (B, N // B),
                   "ri": (B, N // B, N // B), "ri.b": (B, N // B), "lam": (N,), "o": (W, N)}
        out.update({tensor_name(i, "mix", k): v for k, v in mix.items()})
        out[tensor_name(i, "norm", "1")] = (W,)
        if layer.mlp is not None:
            F = layer.mlp.ff
            out[tensor_name(i, "norm", "2")] = (W,)
            out.update({tensor_name(i, "mlp", "gate"): (F, W), tensor_name(i, "mlp", "up"): (F, W), tensor_name(i, "mlp", "down"): (W, F)})
    return out

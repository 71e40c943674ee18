"""Sapasun: its ``config.json`` and the names of its tensors, in terms of the layered decoder (``LayeredConfig``).

Two token mixers (a gated delta rule with a decay per key channel, and chunked grouped-query attention with short convolutions, a
softmax sink, a gate per head and values mixed with the first layer's), an optional squared-relu MLP beside the mixer, two norms of the
same stream per layer, a norm on the embedding and soft-capped logits.
"""
from __future__ import annotations

from .llm_config import PARALLEL_NORM, AttentionSpec, ChannelDeltaSpec, LayeredConfig, LayerSpec, RotarySpec, SquaredReluSpec


def _mixer(kind: str, m: dict):
    heads, kv, dim, vdim, taps = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
    if heads % kv:
        raise ValueError("%d heads do not share %d key / value heads evenly" % (heads, kv))
    if kind == "attention":
        rot = m.get("rot")
        return AttentionSpec(heads, kv, dim, vdim, float(m["scale"]), rotary=RotarySpec(int(rot["dims"]), float(rot["base"])) if rot else None, head_gate=True,
                             chunk=int(m["mask"]["size"]), sink=True, taps=taps, v_mix=bool(m.get("v_mix", False)))
    if kind == "channel_delta":
        return ChannelDeltaSpec(heads, kv, dim, vdim, taps)
    raise ValueError("unknown token mixer '%s'" % kind)


def _mlp(m):
    if m is None:
        return None
    if m["kind"] != "dense":
        raise ValueError("unknown feed-forward '%s'" % m["kind"])
    return SquaredReluSpec(int(m["ff"]))


def read_config(cfg: dict) -> LayeredConfig:
    layers = tuple(LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in cfg["layers"])
    return LayeredConfig("Sapasun", int(cfg["vocab"]), int(cfg["width"]), layers, norm_eps=float(cfg["norm"]["eps"]), block=PARALLEL_NORM, embed_norm=True,
                         logit_softcap=float(cfg["logit_softcap"]))


def tensor_name(layer: int, part: str, key: str) -> str:
    """Name in the checkpoint. ``part``: "mix" / "mlp" / "norm" (key "1" or "2") of a layer; layer -1: "embed", "embed.norm", "final.norm",
    "head"."""
    if layer < 0:
        return key
    return "l%d.norm%s" % (layer, key) if part == "norm" else "l%d.%s.%s" % (layer, part, key)


def tensor_shapes(cfg: LayeredConfig) -> dict:
    """Name -> shape of every tensor of a checkpoint (None: a size that only the tensor gives)."""
    W = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, W), "embed.norm": (W,), "final.norm": (W,), "head": (cfg.vocab_size, W)}
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if isinstance(m, AttentionSpec):
            rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
            mix = {"vmix": (), "sink": (m.heads,), "g": (m.heads, W)}
        else:
            rows = {"q": m.kv_heads * m.dim, "k": m.kv_heads * m.dim, "v": m.heads * m.vdim}
            mix = {"b": (m.heads, W), "A_log": (m.heads,), "norm": (m.vdim,), "a1": (m.decay_rank or None, W), "a2": (m.heads * m.dim, m.decay_rank or None),
                   "dt_bias": (m.heads * m.dim,), "g1": (m.gate_rank or None, W), "g2": (m.heads * m.vdim, m.gate_rank or None)}
        for k, n in rows.items():
            mix[k], mix[k + ".conv"] = (n, W), (n, m.taps)
        mix["o"] = (W, m.heads * m.vdim)
        out.update({tensor_name(i, "mix", k): v for k, v in mix.items()})
        out[tensor_name(i, "norm", "1")] = (W,)
        if layer.mlp is not None:
            F = layer.mlp.ff
            out[tensor_name(i, "norm", "2")] = (W,)
            out.update({tensor_name(i, "mlp", "up"): (F, W), tensor_name(i, "mlp", "down"): (W, F)})
    return out

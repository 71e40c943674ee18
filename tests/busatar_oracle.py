"""Plain, slow implementation of the Busatar decoder: one function per mechanism, whole sequences only, no cache.

The oracle of the serving program's tests. It shares no code with the product: it takes the configuration as the plain
dictionary that ``config.json`` holds and the weights as a name -> tensor dictionary, and computes in the precision of
``dtype`` (float64 by default), one request at a time.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch


def write_model(folder, cfg, weights):
    """config.json + model.safetensors (bfloat16) from a configuration and its weights."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for name, t in weights.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    text = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for b in blobs:
            f.write(b)


def random_weights(cfg, seed=0, gain=1.0):
    """Random weights (values exact in bfloat16, returned as float32) of the shapes that ``cfg`` asks for."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape):
        return torch.randn(*shape, generator=g) * (gain / math.sqrt(shape[-1]))

    def vec(n, mean=0.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": torch.randn(V, W, generator=g)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, t = "l%d." % i, layer["mixer"], layer["type"]
        w[p + "norm1"] = vec(W)
        if t == "attention":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"] = mat(H * D, W), mat(G * D, W), mat(G * Dv, W)
            w[p + "mix.q.norm"], w[p + "mix.k.norm"] = vec(D, 1.0), vec(D, 1.0)
            w[p + "mix.g"], w[p + "mix.o"] = mat(H * Dv, W), mat(W, H * Dv)
        elif t == "latent_attention":
            H, D, R, Dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[p + "mix.q"], w[p + "mix.dkv"], w[p + "mix.dkv.norm"] = mat(H * (D + R), W), mat(C + R, W), vec(C, 1.0)
            w[p + "mix.uk"], w[p + "mix.uv"], w[p + "mix.o"] = mat(H * D, C), mat(H * Dv, C), mat(W, H * Dv)
        elif t == "rglru":
            N, B, taps = m["width"], m["blocks"], m["conv"]
            w[p + "mix.y"], w[p + "mix.y.b"], w[p + "mix.x"], w[p + "mix.x.b"] = mat(N, W), vec(N), mat(N, W), vec(N)
            w[p + "mix.conv"], w[p + "mix.conv.b"] = torch.randn(N, taps, generator=g) / math.sqrt(taps), vec(N)
            for k in ("ra", "ri"):
                w[p + "mix." + k], w[p + "mix." + k + ".b"] = mat(B, N // B, N // B), vec(N).reshape(B, N // B)
            w[p + "mix.lam"], w[p + "mix.o"] = vec(N, -3.0, 1.0), mat(W, N)
        else:
            raise ValueError(t)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            w[p + "norm2"] = vec(W)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(F, W), mat(F, W), mat(W, F)
    w["final.norm"], w["head"] = vec(W), mat(V, W)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def yarn(rot):
    """(frequencies, multiplier of cos and sin) of a rotary table with an optional YaRN 'scaling' entry."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def dim_of(turns):
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim_of(s["fast"])), 0), min(math.ceil(dim_of(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot, start=0):
    """x [tokens, heads, dim]: the first rot.dims dimensions turned by the position, halves paired."""
    n = rot["dims"]
    f, mult = yarn(rot)
    a = torch.arange(start, start + x.shape[0], dtype=torch.float64)[:, None] * f
    cos, sin = (a.cos() * mult).to(x.dtype)[:, None], (a.sin() * mult).to(x.dtype)[:, None]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., n:]], -1)


def window_softmax(q, k, v, scale, window):
    """q [T, H, D], k [T, H, D], v [T, H, Dv]: each position attends to itself and the window - 1 positions before it."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & (i - j < window)
    s = s.masked_fill(~seen, float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def attention(h, w, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w["q"].T).reshape(T, H, D), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).reshape(T, G, D), eps) * w["k.norm"]
    v = (h @ w["v"].T).reshape(T, G, Dv)
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    o = window_softmax(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, H * Dv)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def latent_attention(h, w, m, eps):
    T, H, D, R, Dv, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).reshape(T, H, D + R)
    down = h @ w["dkv"].T
    c = rms(down[:, :C], eps) * w["dkv.norm"]
    kr = rotate(down[:, None, C:], m["rot"])
    q = torch.cat([q[..., :D], rotate(q[..., D:], m["rot"])], -1)
    k = torch.cat([(c @ w["uk"].T).reshape(T, H, D), kr.expand(T, H, R)], -1)
    v = (c @ w["uv"].T).reshape(T, H, Dv)
    return window_softmax(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, H * Dv) @ w["o"].T


def causal_conv(x, taps, bias):
    """x [T, N], taps [N, n]: the last tap meets the current token, zeros come before the first."""
    T, n = x.shape[0], taps.shape[1]
    x = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    return sum(x[j:j + T] * taps[:, j] for j in range(n)) + bias


def lru_scan(u, r, i, lam):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); returns S for every token."""
    log_a = -8 * r * torch.nn.functional.softplus(lam)
    a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * u
    s, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        s = a[t] * s + b[t]
        out.append(s)
    return torch.stack(out)


def block_gate(u, w, b):
    """sigmoid of a block-diagonal linear layer: w [blocks, out, in], b [blocks, out]."""
    T, B = u.shape[0], w.shape[0]
    return torch.sigmoid(torch.einsum("tbi,boi->tbo", u.reshape(T, B, -1), w) + b).reshape(T, -1)


def rglru(h, w, m, eps):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    s = lru_scan(u, block_gate(u, w["ra"], w["ra.b"]), block_gate(u, w["ri"], w["ri.b"]), w["lam"])
    return (s * y) @ w["o"].T


def limited_glu(h, w, m):
    L = m["limit"]
    g = torch.clamp(h @ w["gate"].T, max=L)
    u = torch.clamp(h @ w["up"].T, -L, L)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w["down"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "rglru": rglru}


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=torch.float64, stop=None):
    """(logits [T, vocab], [residual stream after every layer]) of one sequence."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    layers = []
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % i

        def part(kind):
            pre = p + kind + "."
            return {k[len(pre):]: v for k, v in w.items() if k.startswith(pre)}

        x = zero_centred_norm(alpha * x + MIXERS[layer["type"]](x, part("mix"), layer["mixer"], eps), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = zero_centred_norm(alpha * x + limited_glu(x, part("mlp"), layer["mlp"]), w[p + "norm2"], eps)
        layers.append(x)
    return zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T, layers


@torch.no_grad()
def generate(cfg, weights, prompt, n):
    """Greedy continuation; also the gap between the best and the second logit of every step."""
    ids, gaps = list(prompt), []
    for _ in range(n):
        top = forward(cfg, weights, ids)[0][-1].topk(2).values
        gaps.append(float(top[0] - top[1]))
        ids.append(int(forward(cfg, weights, ids)[0][-1].argmax()))
    return ids[len(prompt):], gaps

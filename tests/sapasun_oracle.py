"""Plain, slow implementation of the Sapasun decoder: one function per mechanism, whole sequences only, no cache.

The oracle of the serving program's tests. It shares no code with the product: it takes the configuration as the plain
dictionary that ``config.json`` holds and the weights as a name -> tensor dictionary, and computes in the precision of
``dtype`` (float64 by default), one request at a time.
"""
from __future__ import annotations

import math

import torch


def random_weights(cfg, seed=0, gain=1.0):
    """Random weights (values exact in bfloat16, returned as float32) of the shapes that ``cfg`` asks for. The gains of queries and
    keys are such that attention is peaked and single keys matter."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, by=1.0):
        return torch.randn(*shape, generator=g) * (gain * by / math.sqrt(shape[-1]))

    def vec(n, mean=0.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    def taps(n, k):
        return torch.randn(n, k, generator=g) / math.sqrt(k)

    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": torch.randn(V, W, generator=g), "embed.norm": vec(W, 1.0)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, t = "l%d." % i, layer["mixer"], layer["type"]
        H, G, D, Dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        w[p + "norm1"] = vec(W, 1.0)
        if t == "channel_delta":
            rows = {"q": G * D, "k": G * D, "v": H * Dv}
            R = 8 + 4 * i                                    # rank of the two-step projections: only the shapes give it
            w[p + "mix.a1"], w[p + "mix.a2"] = mat(R, W), mat(H * D, R)
            w[p + "mix.g1"], w[p + "mix.g2"] = mat(R + 4, W), mat(H * Dv, R + 4)
            w[p + "mix.b"], w[p + "mix.A_log"], w[p + "mix.dt_bias"] = mat(H, W), vec(H, 0.0, 0.5), vec(H * D, -3.0, 1.0)
            w[p + "mix.norm"] = vec(Dv, 1.0)
        elif t == "attention":
            rows = {"q": H * D, "k": G * D, "v": G * Dv}
            w[p + "mix.g"], w[p + "mix.sink"], w[p + "mix.vmix"] = mat(H, W), vec(H, 1.0, 1.0), torch.tensor(0.3 + 0.1 * (i % 5))
        else:
            raise ValueError(t)
        for k, n in rows.items():
            w[p + "mix." + k], w[p + "mix." + k + ".conv"] = mat(n, W, by=1.5), taps(n, K)
        w[p + "mix.o"] = mat(W, H * Dv)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            w[p + "norm2"], w[p + "mlp.up"], w[p + "mlp.down"] = vec(W, 1.0), mat(F, W), mat(W, F)
    w["final.norm"], w["head"] = vec(W, 1.0), mat(V, W, by=4.0)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def causal_conv(u, taps):
    """u [T, N], taps [N, n]: the last tap meets the current token, zeros come before the first."""
    T, n = u.shape[0], taps.shape[1]
    u = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=u.dtype), u])
    return sum(u[j:j + T] * taps[:, j] for j in range(n))


def silu(z):
    return z * torch.sigmoid(z)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def rotate(x, rot):
    """x [tokens, heads, dim]: the first rot.dims dimensions turned by the position, halves paired."""
    n = rot["dims"]
    f = torch.tensor([rot["base"] ** (-2 * i / n) for i in range(n // 2)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * f
    cos, sin = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., n:]], -1)


def chunk_sink_softmax(q, k, v, scale, chunk, sink):
    """q [T, H, D], k [T, H, D], v [T, H, Dv], sink [H]: a position attends to itself and what comes before it in its chunk; the
    sink takes part in the denominator only."""
    T, H = q.shape[0], q.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    s = s.masked_fill(~((j <= i) & (i // chunk == j // chunk)), float("-inf"))
    s = torch.cat([s, sink[:, None, None].expand(H, T, 1)], -1)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1)[..., :T], v)


def attention(h, w, m, eps, shared):
    """``shared``: values of the first layer that mixes values (empty until that layer has run)."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(causal_conv(h @ w["q"].T, w["q.conv"]).reshape(T, H, D), m["rot"])
    k = rotate(causal_conv(h @ w["k"].T, w["k.conv"]).reshape(T, G, D), m["rot"])
    v = causal_conv(h @ w["v"].T, w["v.conv"])
    if m.get("v_mix"):
        if shared:
            v = (1 - w["vmix"]) * v + w["vmix"] * shared[0]
        else:
            shared.append(v)
    v = v.reshape(T, G, Dv)
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    o = chunk_sink_softmax(q, k, v, m["scale"], m["mask"]["size"], w["sink"])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * Dv) @ w["o"].T


def delta_scan(q, k, v, g, beta):
    """q, k, g [T, H, D], v [T, H, Dv], beta [T, H]: decay the rows of the state, replace what it holds under the key by a step of
    beta towards the value, read with the query. Returns [T, H, Dv]."""
    S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), []
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def channel_delta(h, w, m, eps, shared):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(silu(causal_conv(h @ w["q"].T, w["q.conv"])).reshape(T, G, D)) * D ** -0.5
    k = unit(silu(causal_conv(h @ w["k"].T, w["k.conv"])).reshape(T, G, D))
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).reshape(T, H, Dv)
    dt = torch.nn.functional.softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).reshape(T, H, D)
    g = torch.exp(-torch.exp(w["A_log"])[:, None] * dt)
    beta = torch.sigmoid(h @ w["b"].T)
    o = delta_scan(q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1), v, g, beta)
    o = rms_norm(o, w["norm"], eps).reshape(T, H * Dv) * torch.sigmoid((h @ w["g1"].T) @ w["g2"].T)
    return o @ w["o"].T


def squared_relu_mlp(h, w):
    return torch.relu(h @ w["up"].T) ** 2 @ w["down"].T


def soft_cap(logits, cap):
    return cap * torch.tanh(logits / cap)


MIXERS = {"attention": attention, "channel_delta": channel_delta}


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=torch.float64):
    """(logits [T, vocab], [residual stream after every layer]) of one sequence."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = rms_norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    layers, shared = [], []
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % i

        def part(kind):
            pre = p + kind + "."
            return {k[len(pre):]: v for k, v in w.items() if k.startswith(pre)}

        y = MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), part("mix"), layer["mixer"], eps, shared)
        if layer["mlp"] is not None:
            y = y + squared_relu_mlp(rms_norm(x, w[p + "norm2"], eps), part("mlp"))
        x = x + y
        layers.append(x)
    return soft_cap(rms_norm(x, w["final.norm"], eps) @ w["head"].T, cfg["logit_softcap"]), layers


@torch.no_grad()
def generate(cfg, weights, prompt, n):
    """Greedy continuation; also the gap between the best and the second logit of every step."""
    ids, gaps = list(prompt), []
    for _ in range(n):
        last = forward(cfg, weights, ids)[0][-1]
        top = last.topk(2)
        gaps.append(float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], gaps

"""Each mechanism of the layered decoders' kernels against the plain oracle (tests/busatar_oracle.py), on inputs that make a wrong
key, a window that is one position off or a lost state visible."""
import math

import pytest
import torch

import busatar_oracle as oracle
from layered_kernel_helpers import PagedBatch

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def up(n, m):
    return (n + m - 1) // m * m


def randn(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).float()


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all()
    err = (got - want).abs().max() / want.abs().max().clamp_min(1e-6)
    assert err < tol, float(err)


def k():
    from openvino_b200.ops import cuda as K
    return K


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [40, 200, 1030, 5000])
def test_sum_then_norm(dtype, width):
    K, rows, pitch = k(), 7, up(width, 64)
    h, y, w = randn(rows, width, seed=1), randn(rows, width, seed=2, scale=3.0), randn(width, seed=3, scale=0.3)
    dev = lambda t: torch.nn.functional.pad(t, (0, pitch - width)).cuda()
    hd, yd, wd = dev(h), dev(y), torch.nn.functional.pad(w, (0, up(width, 4) - width)).cuda()
    x = torch.zeros(rows, pitch, dtype=dtype, device="cuda")
    K.sum_rmsnorm(hd, wd, 1e-3, width, y=yd, alpha=2.5, w_offset=1.0, h_out=hd, x_out=x)
    want = oracle.zero_centred_norm(2.5 * h.double() + y.double(), w.double(), 1e-3)
    close(hd[:, :width], want, 2e-6)
    close(x[:, :width], want, 2e-6 if dtype == torch.float32 else 5e-3)
    assert (x[:, width:] == 0).all() and (hd[:, width:] == 0).all()
    # rows picked out, plain weight, nothing added; a tiny row shows where eps stands
    h[3] *= 1e-3
    pick = torch.tensor([3, 0, 3], dtype=torch.int32, device="cuda")
    out = torch.zeros(3, pitch, dtype=torch.float32, device="cuda")
    K.sum_rmsnorm(dev(h), wd, 1e-3, width, x_out=out, row_idx=pick)
    close(out[:, :width], oracle.rms(h[[3, 0, 3]].double(), 1e-3) * w.double(), 2e-6)


@pytest.mark.parametrize("limit", [0.7, 2.0])
@pytest.mark.parametrize("ff", [64, 100, 448])
def test_limited_glu(limit, ff):
    K, rows, width = k(), 9, 128
    x, gate, up_w = randn(rows, width, seed=1), randn(ff, width, seed=2, scale=0.3), randn(ff, width, seed=3, scale=0.3)
    x, gate, up_w = [t.to(torch.bfloat16).float() for t in (x, gate, up_w)]
    eye = torch.eye(ff, dtype=torch.float64)
    want = oracle.limited_glu(x.double(), {"gate": gate.double(), "up": up_w.double(), "down": eye}, {"limit": limit})
    assert (x @ gate.T > limit).any() and (x @ up_w.T).abs().max() > limit
    fp = up(ff, 64)
    pad = lambda t: torch.nn.functional.pad(t, (0, 0, 0, fp - ff)).cuda()
    gu = torch.zeros(rows, 2 * fp, device="cuda")
    K.gemm(x.cuda(), K.PackedWeight(K.W_F32, torch.cat([pad(gate), pad(up_w)]), 2 * fp, width), out=gu)
    out = torch.zeros(rows, fp, device="cuda")
    close(K.glu_limited(gu, out, ff, fp, limit)[:, :ff], want, 1e-5)
    # the bf16 form in the epilogue of the product
    w = K.PackedWeight.from_dense(K.interleave_gate_up(pad(gate), pad(up_w)).to(torch.bfloat16))
    got = K.gemm(x.cuda().to(torch.bfloat16), w, act=K.ACT_GLU_LIMITED, glu=(limit, 1.702, 1.0))
    close(got[:, :ff], want, 1e-2)
    assert (got[:, ff:] == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("G,N,Kd,pitch,opitch", [(3, 40, 24, 32, 48), (5, 200, 96, 112, 208), (1, 64, 64, 64, 64), (6, 128, 130, 144, 128)])
def test_block_diagonal_product(dtype, G, N, Kd, pitch, opitch):
    K = k()
    for T in (1, 5, 70, 300):
        x, w = randn(T, G * pitch, seed=T, dtype=dtype), randn(G, N, Kd, seed=2, dtype=dtype)
        out = torch.full((T, G * opitch), 7.0, dtype=dtype, device="cuda")
        K.gemm_block_diag(x.cuda().to(dtype), K.BlockDiagWeight(w.cuda().to(dtype)), out, pitch, opitch)
        want = torch.einsum("tgk,gnk->tgn", x.double().reshape(T, G, pitch)[..., :Kd], w.double())
        close(out.reshape(T, G, opitch)[..., :N], want, 1e-5 if dtype == torch.float32 else 1e-2)
        assert (out.reshape(T, G, opitch)[..., N:] == 7).all()
        if dtype == torch.bfloat16:
            out32 = torch.zeros(T, G * opitch, device="cuda")
            K.gemm_block_diag(x.cuda().to(dtype), K.BlockDiagWeight(w.cuda().to(dtype)), out32, pitch, opitch)
            close(out32.reshape(T, G, opitch)[..., :N], want, 1e-5)


@pytest.mark.parametrize("act", [0, 5])
def test_fp32_product(act):
    K = k()
    for T, N, Kd in ((1, 3, 5), (67, 130, 70), (128, 64, 256)):
        x, w, b = randn(T, Kd, seed=1), randn(N, Kd, seed=2), randn(N, seed=3)
        got = K.gemm(x.cuda(), K.PackedWeight(K.W_F32, w.cuda(), N, Kd, bias=b.cuda()), act=act)
        want = x.double() @ w.double().T + b.double()
        close(got, oracle.gelu_tanh(want) if act == 5 else want, 2e-6)


ROT = [None, dict(dims=16, base=1e4), dict(dims=24, base=5e5, scaling=dict(factor=4.0, original=64, fast=8.0, slow=1.0)),
       dict(dims=32, base=1e4, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0))]


def rotation(rot):
    from openvino_b200.models.busatar import _rotary
    from openvino_b200.runtime.layered_llm import _Rotation
    return _Rotation(_rotary(rot) if rot else None, "cuda")


def rope(rot, positions):
    r = rotation(rot)
    if not r.dims:
        return {}
    table = torch.zeros(positions.numel(), r.dims, device="cuda")
    k().rope_table(positions, r.inv_freq, table, r.mult)
    return dict(rot_dims=r.dims, rope=table)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rot", ROT[:3])
@pytest.mark.parametrize("norm", [True, False])
def test_heads_prepare(dtype, rot, norm):
    K, H, G, D, Dv = k(), 6, 2, 40, 24
    dk, dv, eps = up(D, 16), up(Dv, 16), 1e-3
    pb = PagedBatch([(0, 5), (37, 1), (14, 20)])
    q, kk, v = randn(pb.T, H, D, seed=1, dtype=dtype), randn(pb.T, G, D, seed=2, scale=4.0, dtype=dtype), randn(pb.T, G, Dv, seed=3, dtype=dtype)
    wq, wk = randn(D, seed=4), randn(D, seed=5)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).reshape(pb.T, -1)
    proj = torch.cat([pad(q, dk), pad(kk, dk), pad(v, dv)], 1).cuda().to(dtype)
    kc, vc = torch.zeros(pb.num_blocks, G, 16, dk, dtype=dtype, device="cuda"), torch.zeros(pb.num_blocks, G, 16, dv, dtype=dtype, device="cuda")
    K.heads_prepare(proj=proj, k_cache=kc, v_cache=vc, q_norm=wq.cuda() if norm else None, k_norm=wk.cuda() if norm else None, positions=pb.positions,
                    slot_map=pb.slot_map, T=pb.T, H=H, G=G, D=D, Dv=Dv, dk_pad=dk, dv_pad=dv, ldp=proj.stride(0), k_off=H * dk, v_off=(H + G) * dk,
                    block_size=16, dtype=K.storage_type(dtype), eps=eps, **rope(rot, pb.positions))
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    for b, (past, n) in enumerate(pb.spans):
        rows = slice(pb.begins[b], pb.begins[b] + n)
        qq, kw = q[rows].double(), kk[rows].double()
        if norm:
            qq, kw = oracle.rms(qq, eps) * wq.double(), oracle.rms(kw, eps) * wk.double()
        if rot:
            qq, kw = oracle.rotate(qq, rot, past), oracle.rotate(kw, rot, past)
        close(proj[rows, :H * dk].reshape(n, H, dk)[..., :D], qq, tol)
        for i in range(n):
            s = pb.slot(b, past + i)
            close(kc[s // 16, :, s % 16, :D], kw[i], tol)
            close(vc[s // 16, :, s % 16, :Dv], v[rows][i], 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rot", ROT[1:])
def test_latent_prepare(dtype, rot):
    K, H, D, R, C, eps = k(), 3, 20, 32, 72, 1e-3
    dp, rp, cp = up(D, 16), up(R, 16), up(C, 16)
    pb = PagedBatch([(0, 5), (3000, 1), (14, 9)])
    q, c, kr = randn(pb.T, H, D + R, seed=1, dtype=dtype), randn(pb.T, C, seed=2, scale=5.0, dtype=dtype), randn(pb.T, R, seed=3, dtype=dtype)
    w = randn(C, seed=4)
    qp = torch.zeros(pb.T, H, dp + rp)
    qp[..., :D], qp[..., dp:dp + R] = q[..., :D], q[..., D:]
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))
    proj = torch.cat([qp.reshape(pb.T, -1), pad(c, cp), pad(kr, rp)], 1).cuda().to(dtype)
    cache = torch.zeros(pb.num_blocks, 16, cp + rp, dtype=dtype, device="cuda")
    out = torch.zeros(pb.T, H * (cp + rp), dtype=dtype, device="cuda")
    K.latent_prepare(proj=proj, q_rot=out[:, cp:], cache=cache, c_norm=w.cuda(), positions=pb.positions, slot_map=pb.slot_map, T=pb.T, H=H, C=C, R=R,
                     q_pitch=dp + rp, q_rot_off=dp, c_off=H * (dp + rp), kr_off=H * (dp + rp) + cp, ldp=proj.stride(0), ld_qr=out.stride(0), qr_pitch=cp + rp,
                     row_pitch=cp + rp, key_off=cp, block_size=16, dtype=K.storage_type(dtype), eps=eps, **rotation(rot).args())
    tol = 2e-4 if dtype == torch.float32 else 1e-2           # fp32 angles of a few thousand turns
    for b, (past, n) in enumerate(pb.spans):
        rows = slice(pb.begins[b], pb.begins[b] + n)
        close(out[rows].reshape(n, H, cp + rp)[..., cp:cp + R], oracle.rotate(q[rows][..., D:].double(), rot, past), tol)
        lat, key = oracle.rms(c[rows].double(), eps) * w.double(), oracle.rotate(kr[rows][:, None].double(), rot, past)[:, 0]
        for i in range(n):
            s = pb.slot(b, past + i)
            close(cache[s // 16, s % 16, :C], lat[i], tol)
            close(cache[s // 16, s % 16, cp:cp + R], key[i], tol)


def attend(q, kv, vv, spans, scale, window):
    """Oracle attention of the new tokens of every sequence (whole sequences in, heads already expanded)."""
    out = []
    for x, a, c, (past, n) in zip(q, kv, vv, spans):
        out.append(oracle.window_softmax(x.double(), a.double(), c.double(), scale, window or 10 ** 9)[past:])
    return torch.cat(out)


def planted(T, H, D, window, seed, reach):
    """Queries that each look for one key: ``reach`` = how far back (window - 1 is just inside, window just outside)."""
    key = torch.nn.functional.normalize(randn(T, H, D, seed=seed), dim=-1)
    q = torch.stack([key[max(0, i - reach)] for i in range(T)]) * 12.0
    return q.to(torch.bfloat16).float(), key.to(torch.bfloat16).float()


SIZES = [(4, 4, 32, 32), (6, 2, 40, 24), (8, 1, 96, 64), (6, 6, 64, 128), (12, 1, 128, 128), (3, 3, 192, 96), (2, 2, 160, 112), (9, 3, 256, 256), (32, 2, 64, 64),
         (2, 1, 320, 40)]
SPANS = [[(0, 130), (0, 1), (0, 45)], [(70, 2), (0, 17), (33, 64), (150, 1)], [(0, 1), (31, 1), (32, 1), (200, 1), (129, 1)]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("which", [0, 1, 2])
def test_window_attention(dtype, sizes, which):
    K, (H, G, D, Dv), spans = k(), sizes, SPANS[which]
    dk, dv, pb = up(D, 16), up(Dv, 16), PagedBatch(SPANS[which], seed=which)
    for window in (1, 16, 33, 128, 0):
        for reach in (max(window - 1, 0) if window else 60, window or 100):
            q, kk, vv = [], [], []
            for b, (p, n) in enumerate(spans):
                a, c = planted(p + n, G, D, window, 10 * b + which, reach)
                q.append(a.repeat_interleave(H // G, 1) + randn(p + n, H, D, seed=b + 50, scale=0.3, dtype=torch.bfloat16))
                q[-1] = q[-1].to(torch.bfloat16).float()
                kk.append(c)
                vv.append(randn(p + n, G, Dv, seed=b + 90, dtype=torch.bfloat16))
            scale, gate = 0.8, randn(pb.T, H * dv, seed=7, dtype=torch.bfloat16)
            want = attend(q, [x.repeat_interleave(H // G, 1) for x in kk], [x.repeat_interleave(H // G, 1) for x in vv], spans, scale, window)
            new = torch.cat([x[p:] for x, (p, _) in zip(q, spans)])
            qd = torch.nn.functional.pad(new, (0, dk - D)).reshape(pb.T, H * dk).cuda().to(dtype)
            out = torch.zeros(pb.T, H * dv, dtype=dtype, device="cuda")
            kc, vc = pb.fill(kk, dk, dtype), pb.fill(vv, dv, dtype)
            ws = torch.empty(1 << 22, device="cuda")
            for gated in (False, True):
                g = dict(gate=gate.cuda().to(dtype), ld_gate=H * dv, gate_head=dv) if gated else {}
                K.window_attention(q=qd, k=kc, v=vc, out=out, Hq=H, Hkv=G, Dk=dk, Dv=Dv, ldq=H * dk, q_head=dk, k_row=dk, v_row=dv, ldo=H * dv, o_head=dv,
                                   window=window, scale=scale, max_context_len=pb.max_ctx, max_q_len=pb.max_q_len, dtype=K.storage_type(dtype), scratch=ws,
                                   scratch_bytes=ws.nbytes, exact=1 if dtype == torch.float32 else 0, **g, **pb.args)
                expect = want * torch.sigmoid(gate.double().reshape(pb.T, H, dv)[..., :Dv]) if gated else want
                close(out.reshape(pb.T, H, dv)[..., :Dv], expect, 1e-5 if dtype == torch.float32 else 1.5e-2)
    K.check_status("window attention")


LATENT = [(4, 32, 16, 48, 64), (6, 64, 16, 48, 112), (3, 40, 8, 24, 72), (20, 128, 64, 128, 256), (40, 96, 32, 112, 512), (5, 160, 64, 32, 128), (2, 16, 8, 16, 600)]


@pytest.mark.parametrize("sizes", LATENT)
@pytest.mark.parametrize("which", [0, 1, 2])
def test_latent_attention_forms(sizes, which):
    """Absorbed form (tensor-core kernel in bf16, exact kernel in fp32) and expanded form against per-head keys and values."""
    K, (H, D, R, Dv, C), spans = k(), sizes, SPANS[which]
    dp, rp, cp, dv = up(D, 16), up(R, 16), up(C, 16), up(Dv, 16)
    pb, row, bf = PagedBatch(spans, seed=which), up(C, 16) + up(R, 16), torch.bfloat16
    uk, uv = randn(H, D, C, seed=1, scale=1 / math.sqrt(C), dtype=bf), randn(H, Dv, C, seed=2, scale=1 / math.sqrt(C), dtype=bf)
    for window in (1, 33, 128, 0):
        for reach in (max(window - 1, 0) if window else 60, window or 100):
            lat, key, q = [], [], []
            for b, (p, n) in enumerate(spans):
                c, r = randn(p + n, C, seed=b + 3, dtype=bf), torch.nn.functional.normalize(randn(p + n, R, seed=b + 4), dim=-1).to(bf).float()
                lat.append(c)
                key.append(r)
                aim = torch.stack([r[max(0, i - reach)] for i in range(p + n)]) * 10.0        # the shared part finds the planted key
                qn = randn(p + n, H, D, seed=b + 5, scale=0.3)
                q.append(torch.cat([qn, aim[:, None].expand(-1, H, -1)], -1).to(bf).float())
            scale = 1.1
            kk = [torch.cat([torch.einsum("tc,hdc->thd", c, uk), r[:, None].expand(-1, H, -1)], -1) for c, r in zip(lat, key)]
            vv = [torch.einsum("tc,hdc->thd", c, uv) for c in lat]
            want = attend(q, kk, vv, spans, scale, window)
            new = torch.cat([x[p:] for x, (p, _) in zip(q, spans)])
            rows = [torch.cat([torch.nn.functional.pad(c, (0, cp - C)), r], -1)[:, None] for c, r in zip(lat, key)]
            ws = torch.empty(1 << 23, device="cuda")
            for dtype in DTYPES:
                pitch = row + 8
                cache = pb.fill(rows, pitch, dtype)
                qd = torch.zeros(pb.T, H, dp + rp)
                qd[..., :D], qd[..., dp:dp + R] = new[..., :D], new[..., D:]
                qd = qd.reshape(pb.T, -1).cuda().to(dtype)
                qa = torch.zeros(pb.T, H * row, dtype=dtype, device="cuda")
                qa.view(pb.T, H, row)[..., cp:cp + R] = new[..., D:].cuda().to(dtype)
                K.gemm_block_diag(qd, K.BlockDiagWeight(uk.transpose(1, 2).cuda().to(dtype)), qa, dp + rp, row)
                lo = torch.zeros(pb.T, H * cp, dtype=dtype, device="cuda")
                K.window_attention(q=qa, k=cache, v=cache, out=lo, Hq=H, Hkv=1, Dk=row, Dv=C, ldq=H * row, q_head=row, k_row=pitch, v_row=pitch, ldo=H * cp, o_head=cp,
                                   window=window, scale=scale, max_context_len=pb.max_ctx, max_q_len=pb.max_q_len, dtype=K.storage_type(dtype), scratch=ws,
                                   scratch_bytes=ws.nbytes, exact=1 if dtype == torch.float32 else 0, **pb.args)
                out = torch.zeros(pb.T, H * dv, dtype=dtype, device="cuda")
                K.gemm_block_diag(lo, K.BlockDiagWeight(uv.cuda().to(dtype)), out, cp, dv)
                close(out.reshape(pb.T, H, dv)[..., :Dv], want, 2e-5 if dtype == torch.float32 else 2.5e-2)
            kh, vh = up(D, 64), up(Dv, 64)
            if kh > 128 or vh > 128 or R > 64:
                continue
            first = [max(0, p - window + 1) // 128 * 128 if window else 0 for p, _ in spans]
            n = sum(p + m - f for (p, m), f in zip(spans, first))
            batch = dict(pb.args, window=window)
            T = batch.pop("T")
            g, begins = torch.zeros(n, up(C, 64), dtype=bf, device="cuda"), torch.zeros(pb.B + 1, dtype=torch.int32, device="cuda")
            K.latent_gather(cache=cache, out=g, kv_rows=begins, rows=n, cols=cp, row_pitch=pitch, out_pitch=g.stride(0), **batch)
            assert torch.equal(g[:, :C].float().cpu(), torch.cat([c[f:] for c, f in zip(lat, first)]))
            wk, wv = torch.nn.functional.pad(uk, (0, g.shape[1] - C, 0, kh - D)), torch.nn.functional.pad(uv, (0, g.shape[1] - C, 0, vh - Dv))
            kv = K.gemm(g, K.PackedWeight.from_dense(torch.cat([wk.reshape(H * kh, -1), wv.reshape(H * vh, -1)]).to(bf).cuda()))
            out = torch.zeros(T, H * dv, dtype=bf, device="cuda")
            K.latent_prefill(q=qd, kv=kv, cache=cache, out=out, kv_rows=begins, T=T, H=H, rows=n, R=R, Dv=dv, ldq=qd.stride(0), q_head=dp + rp, q_rot_off=dp,
                             ld_kv=kv.stride(0), k_head=kh, v_off=H * kh, v_head=vh, row_pitch=pitch, key_off=cp, ldo=H * dv, o_head=dv, scale=scale, **batch)
            close(out.reshape(T, H, dv)[..., :Dv], want, 2.5e-2)
    K.check_status("latent attention")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,blocks,taps", [(64, 2, 4), (120, 3, 3), (96, 1, 1), (320, 8, 2), (40, 5, 8)])
def test_recurrent_block_in_portions(dtype, N, blocks, taps):
    """Convolution, gates and recurrence over prompts cut at all kinds of places; slots are reused without being cleared."""
    K, bw = k(), N // blocks
    bp, lens = up(bw, 16), [150, 1, 7, 33]
    w = {n: randn(*s, seed=i, scale=c, dtype=torch.bfloat16) for i, (n, s, c) in enumerate([
        ("conv", (N, taps), 0.7), ("conv.b", (N,), 0.2), ("ra", (blocks, bw, bw), 0.3), ("ra.b", (blocks, bw), 0.3), ("ri", (blocks, bw, bw), 0.3),
        ("ri.b", (blocks, bw), 0.3), ("lam", (N,), 1.0)])}
    w["lam"] = w["lam"] - 4.0                                 # slow decay: what was lost early is still missing late
    xs = [randn(n, N, seed=20 + b, dtype=torch.bfloat16) for b, n in enumerate(lens)]
    ys = [randn(n, N, seed=40 + b, dtype=torch.bfloat16) for b, n in enumerate(lens)]
    want = []
    for x, y in zip(xs, ys):
        u = oracle.causal_conv(x.double(), w["conv"].double(), w["conv.b"].double())
        u = u.to(dtype).double() if dtype == torch.bfloat16 else u
        gates = [oracle.block_gate(u, w[n].double(), w[n + ".b"].double()) for n in ("ra", "ri")]
        want.append(oracle.lru_scan(u, *gates, w["lam"].double()) * oracle.gelu_tanh(y.double()))
    pad = lambda t: torch.nn.functional.pad(t, (0, 0, 0, bp - bw))
    gw = K.BlockDiagWeight(torch.cat([pad(w["ra"]), pad(w["ri"])], 1).cuda().to(dtype))
    const = dict(gate_b=torch.stack([w["ra.b"].reshape(-1), w["ri.b"].reshape(-1)]).cuda().contiguous(),
                 log_decay=(8 * torch.nn.functional.softplus(w["lam"].double())).float().cuda(), conv_w=w["conv"].t().contiguous().cuda(), conv_b=w["conv.b"].cuda())
    state, conv = torch.full((9, N), 3.0, device="cuda"), torch.full((9, max(taps - 1, 1), N), 3.0, device="cuda")
    slots, at, got = [7, 2, 0, 5], [0] * 4, [[] for _ in lens]
    for cut in ([3, 1, 2, 1], [1, 0, 1, 1], [2, 0, 0, 20], [64, 0, 0, 11], [1, 0, 4, 0], [79, 0, 0, 0]):
        batch = [(b, at[b], n) for b, n in enumerate(cut) if n]
        T = sum(n for _, _, n in batch)
        cat = lambda seqs: torch.cat([seqs[b][s:s + n] for b, s, n in batch]).cuda().to(dtype)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
        begins = [0]
        for _, _, n in batch:
            begins.append(begins[-1] + n)
        x, y = cat(xs), cat(ys)
        u, gates, out = torch.zeros(T, blocks * bp, dtype=dtype, device="cuda"), torch.zeros(T, blocks * 2 * bp, device="cuda"), torch.zeros(T, N, dtype=dtype, device="cuda")
        args = dict(x=x, y=y, u=u, out=out, gates=gates, state=state, conv_state=conv, subsequence_begins=i32(begins), past_lens=i32([s for _, s, _ in batch]),
                    slots=i32([slots[b] for b, _, _ in batch]), B=len(batch), T=T, N=N, taps=taps, bw=bw, ub_pitch=bp, gb_pitch=2 * bp, gi_off=bp, ldx=N, ldy=N,
                    ldu=u.stride(0), ldg=gates.stride(0), ldo=N, max_q_len=max(n for _, _, n in batch), dtype=K.storage_type(dtype), **const)
        K.causal_conv(**args)
        K.gemm_block_diag(u, gw, gates, bp, 2 * bp)
        K.lru_scan(**args)
        for (b, _, n), lo in zip(batch, begins):
            got[b].append(out[lo:lo + n].float().cpu())
            at[b] += n
    assert at == lens
    for g, v in zip(got, want):
        close(torch.cat(g), v, 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("vocab", [37, 480, 5000])
def test_fp32_sampling(vocab):
    K = k()
    x = randn(5, vocab, seed=vocab)
    x[2, vocab - 1] = x[2].max() + 1e-6                       # a gap that bf16 logits could not tell
    assert torch.equal(K.argmax(x.cuda()).cpu(), x.argmax(-1))
    got = K.sample(x.cuda(), 0.7, top_k=1, seed=3)
    assert torch.equal(got.cpu().long(), x.argmax(-1))
    drawn = torch.stack([K.sample(x.cuda(), 1.0, top_k=3, seed=s) for s in range(40)]).cpu().long()
    top = x.topk(3).indices
    assert all(set(drawn[:, r].tolist()) <= set(top[r].tolist()) for r in range(5))

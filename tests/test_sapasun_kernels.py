"""Each mechanism that Sapasun adds to the layered decoders' kernels against the plain oracle (tests/sapasun_oracle.py), on inputs that
make a wrong key, a chunk that begins one position off, a lost sink or a lost state visible."""
import math

import pytest
import torch

import sapasun_oracle as oracle
from layered_kernel_helpers import PagedBatch
from test_layered_kernels import DTYPES, SIZES, close, k, randn, up

pytestmark = pytest.mark.gpu


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [40, 202, 1030, 5000])
def test_two_norms_of_a_sum(dtype, width):
    K, rows, pitch = k(), 7, up(width, 64)
    h, y, w, w2 = (randn(*s, seed=i + 1) for i, s in enumerate([(rows, width), (rows, width), (width,), (width,)]))
    h[2] *= 1e-3
    y[2] *= 1e-3                                                  # a tiny row shows where eps stands
    dev = lambda t: torch.nn.functional.pad(t, (0, pitch - width)).cuda()
    vec = lambda t: torch.nn.functional.pad(t, (0, up(width, 4) - width)).cuda()
    hd, yd = dev(h), dev(y)
    x, x2 = torch.zeros(rows, pitch, dtype=dtype, device="cuda"), torch.zeros(rows, pitch, dtype=dtype, device="cuda")
    tol, s = 2e-6 if dtype == torch.float32 else 5e-3, h.double() + y.double()
    # rows picked out of both summands, which stay as they are
    pick = torch.tensor([3, 2, 6], dtype=torch.int32, device="cuda")
    K.sum_rmsnorm(hd, vec(w), 1e-3, width, y=yd, x_out=x[:3], row_idx=pick)
    close(x[:3, :width], oracle.rms_norm(s[[3, 2, 6]], w.double(), 1e-3), tol)
    K.sum_rmsnorm(hd, vec(w), 1e-3, width, y=yd, s_out=hd, x_out=x, w2=vec(w2), x2_out=x2)
    close(hd[:, :width], s, 1e-6)
    for got, wt in ((x, w), (x2, w2)):
        for r in range(rows):
            close(got[r, :width], oracle.rms_norm(s[r], wt.double(), 1e-3), tol)
        assert (got[:, width:] == 0).all()


@pytest.mark.parametrize("T", [1, 40, 130, 300])
@pytest.mark.parametrize("ff,width", [(100, 128), (448, 320), (256, 2048)])
def test_squared_relu_and_soft_cap_epilogues(T, ff, width):
    K, bf, f32 = k(), torch.bfloat16, torch.float32
    x, w = randn(T, width, seed=1, dtype=bf), randn(ff, width, seed=2, scale=1 / math.sqrt(width), dtype=bf)
    z = x.double() @ w.double().T
    assert z.max() > 1 and z.min() < -1
    full, packed = K.PackedWeight(K.W_F32, w.cuda(), ff, width), K.PackedWeight.from_dense(w.to(bf).cuda())
    close(K.gemm(x.cuda(), full, act=K.ACT_RELU2), torch.relu(z) ** 2, 3e-6)
    close(K.gemm(x.cuda().to(bf), packed, act=K.ACT_RELU2), torch.relu(z) ** 2, 5e-3)
    for cap in (0.7, 30.0):
        close(K.gemm(x.cuda(), full, act=K.ACT_SOFTCAP, cap=cap), oracle.soft_cap(z, cap), 3e-6)
        out = torch.zeros(T, ff, dtype=f32, device="cuda")
        close(K.gemm(x.cuda().to(bf), packed, out=out, out_f32=True, act=K.ACT_SOFTCAP, cap=cap), oracle.soft_cap(z, cap), 1e-5)


def test_angle_table_far_out():
    K = k()
    pos = torch.tensor([0, 1, 77, 4096, 60000], dtype=torch.int32)
    f = torch.tensor([250.0 ** (-2 * i / 24) for i in range(12)])
    table = torch.zeros(5, 24, device="cuda")
    K.rope_table(pos.cuda(), f.cuda(), table, 1.0)
    a = (pos[:, None].float() * f).double()                    # fp32 angles
    close(table.view(5, 12, 2), torch.stack([a.cos(), a.sin()], -1), 1e-6)


# ------------------------------------------------------------------------------------------------ chunks, sinks, gates
def chunk_lookers(T, H, D, chunk, seed, inside):
    """Queries that each look for one key: the first of their own chunk, or the last of the chunk before (which must not be found)."""
    key = torch.nn.functional.normalize(randn(T, H, D, seed=seed), dim=-1)
    aim = [i // chunk * chunk - (0 if inside else 1) for i in range(T)]
    q = torch.stack([key[max(0, a)] for a in aim]) * 12.0
    return q.to(torch.bfloat16).float(), key.to(torch.bfloat16).float()


SPANS = [[(0, 150), (0, 1), (0, 45)], [(70, 2), (0, 17), (33, 64), (150, 1), (31, 3)], [(0, 1), (31, 1), (32, 1), (200, 1), (127, 1), (128, 1)]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("which", [0, 1, 2])
def test_chunked_attention_with_sinks_and_head_gates(dtype, sizes, which):
    K, (H, G, D, Dv), spans = k(), sizes, SPANS[which]
    dk, dv, pb = up(D, 16), up(Dv, 16), PagedBatch(SPANS[which], seed=which)
    sink = torch.linspace(-3.0, 11.0, H)                        # from next to nothing to most of the weight
    gate = randn(pb.T, H + 3, seed=7, dtype=torch.bfloat16)     # an odd pitch: one number per head needs no alignment
    ws = torch.empty(1 << 22, device="cuda")
    for chunk in (1, 16, 33, 128, 300):
        for inside in (True, False):
            q, kk, vv, want, plain = [], [], [], [], []
            for b, (p, n) in enumerate(spans):
                a, c = chunk_lookers(p + n, G, D, chunk, 10 * b + which, inside)
                x = (a.repeat_interleave(H // G, 1) + randn(p + n, H, D, seed=b + 50, scale=0.3)).to(torch.bfloat16).float()
                v = randn(p + n, G, Dv, seed=b + 90, dtype=torch.bfloat16)
                rep = lambda t: t.repeat_interleave(H // G, 1).double()
                want.append(oracle.chunk_sink_softmax(x.double(), rep(c), rep(v), 0.8, chunk, sink.double())[p:])
                plain.append(oracle.chunk_sink_softmax(x.double(), rep(c), rep(v), 0.8, chunk, torch.full((H,), -1e9).double())[p:])
                q.append(x[p:])
                kk.append(c)
                vv.append(v)
            qd = torch.nn.functional.pad(torch.cat(q), (0, dk - D)).reshape(pb.T, H * dk).cuda().to(dtype)
            out, kc, vc = torch.zeros(pb.T, H * dv, dtype=dtype, device="cuda"), pb.fill(kk, dk, dtype), pb.fill(vv, dv, dtype)

            def run(**kw):
                K.window_attention(q=qd, k=kc, v=vc, out=out, Hq=H, Hkv=G, Dk=dk, Dv=Dv, ldq=H * dk, q_head=dk, k_row=dk, v_row=dv, ldo=H * dv, o_head=dv, window=0,
                                   chunk=chunk, scale=0.8, max_context_len=pb.max_ctx, max_q_len=pb.max_q_len, dtype=K.storage_type(dtype), scratch=ws,
                                   scratch_bytes=ws.nbytes, exact=1 if dtype == torch.float32 else 0, **kw, **pb.args)
                return out.reshape(pb.T, H, dv)[..., :Dv]
            tol, want, plain = 1e-5 if dtype == torch.float32 else 1.5e-2, torch.cat(want), torch.cat(plain)
            assert (want - plain).abs().max() > 0.2 * plain.abs().max()
            close(run(), plain, tol)
            close(run(sink=sink.cuda()), want, tol)
            g = gate.cuda().to(dtype)
            close(run(sink=sink.cuda(), gate=g[:, 1:], ld_gate=H + 3, gate_head=1, gate_scalar=1),
                  want * torch.sigmoid(gate.double()[:, 1:H + 1, None]), tol)
    K.check_status("chunked attention")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_chunks_are_split_over_ctas(dtype):
    """A decode batch whose chunk spans several splits: the sink counts once, whatever their number."""
    K, H, G, D, chunk, ctx = k(), 8, 2, 64, 3000, [2999, 3000, 3001, 5900]
    pb = PagedBatch([(c, 1) for c in ctx], seed=3)
    sink = torch.linspace(-2.0, 8.0, H)
    q, kk, vv, want = [], [], [], []
    for b, c in enumerate(ctx):
        x, a, v = randn(c + 1, H, D, seed=b, scale=2.0, dtype=torch.bfloat16), randn(c + 1, G, D, seed=b + 10, dtype=torch.bfloat16), \
            randn(c + 1, G, D, seed=b + 20, dtype=torch.bfloat16)
        lo = c // chunk * chunk
        rep = lambda t: t[lo:].repeat_interleave(H // G, 1).double()
        s = torch.cat([torch.einsum("hd,jhd->hj", x[-1].double(), rep(a)) * 0.3, sink.double()[:, None]], 1)
        want.append(torch.einsum("hj,jhd->hd", torch.softmax(s, -1)[:, :-1], rep(v)))
        q.append(x[-1:])
        kk.append(a)
        vv.append(v)
    for scratch in (1 << 22, 16):                                # with and without room for splits
        ws, out = torch.empty(scratch, device="cuda"), torch.zeros(pb.T, H * D, dtype=dtype, device="cuda")
        K.window_attention(q=torch.cat(q).reshape(pb.T, H * D).cuda().to(dtype), k=pb.fill(kk, D, dtype), v=pb.fill(vv, D, dtype), out=out, Hq=H, Hkv=G, Dk=D, Dv=D,
                           ldq=H * D, q_head=D, k_row=D, v_row=D, ldo=H * D, o_head=D, window=0, chunk=chunk, sink=sink.cuda(), scale=0.3, max_context_len=pb.max_ctx,
                           max_q_len=1, dtype=K.storage_type(dtype), scratch=ws, scratch_bytes=ws.nbytes, exact=1 if dtype == torch.float32 else 0, **pb.args)
        close(out.reshape(pb.T, H, D), torch.stack(want), 1e-5 if dtype == torch.float32 else 1.5e-2)


# ------------------------------------------------------------------------------------------------ state in portions
LENS = [150, 1, 7, 33]
CUTS = ([3, 1, 2, 1], [1, 0, 1, 1], [2, 0, 0, 20], [64, 0, 0, 11], [1, 0, 4, 0], [1, 0, 0, 0], [78, 0, 0, 0])


class Portions:
    """Four sequences that arrive in the portions of CUTS; their slots hold rubbish at first. Yields what a kernel call needs."""

    def __init__(self):
        self.slots, self.at = [7, 2, 0, 5], [0] * 4

    def __iter__(self):
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
        for cut in CUTS:
            batch = [(b, self.at[b], n) for b, n in enumerate(cut) if n]
            begins = [0]
            for _, _, n in batch:
                begins.append(begins[-1] + n)
            args = dict(subsequence_begins=i32(begins), past_lens=i32([s for _, s, _ in batch]), slots=i32([self.slots[b] for b, _, _ in batch]), B=len(batch),
                        T=begins[-1], max_q_len=max(n for _, _, n in batch))
            yield batch, begins, args
            for b, _, n in batch:
                self.at[b] += n
        assert self.at == LENS


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv,rot,taps", [(4, 2, 32, 48, 16, 4), (6, 1, 64, 32, 64, 3), (3, 3, 22, 13, 10, 2), (2, 1, 128, 128, 8, 1), (4, 2, 40, 24, 0, 6),
                                               (2, 1, 160, 144, 32, 3)])
def test_short_convolution_rotation_and_value_mixing(dtype, H, G, D, Dv, rot, taps):
    """Queries and cache rows of prompts cut at all kinds of places; convolution inputs of earlier steps come from the ring."""
    K, bf, lam = k(), torch.bfloat16, 0.3125
    dk, dv, r = up(D, 16), up(Dv, 16), dict(dims=rot, base=800.0)
    cols = {"q": (H, D, dk), "k": (G, D, dk), "v": (G, Dv, dv)}
    u = {n: [randn(L, h * d, seed=10 * i + j, dtype=bf) for j, L in enumerate(LENS)] for i, (n, (h, d, _)) in enumerate(cols.items())}
    w = {n: randn(h * d, taps, seed=50 + i, dtype=bf) for i, (n, (h, d, _)) in enumerate(cols.items())}
    first = [randn(L, G * Dv, seed=80 + j, dtype=bf) for j, L in enumerate(LENS)]
    want = {n: [oracle.causal_conv(x.double(), w[n].double()).reshape(len(x), h, d) for x in u[n]] for n, (h, d, _) in cols.items()}
    if rot:
        for n in ("q", "k"):
            want[n] = [oracle.rotate(x, r) for x in want[n]]
    pads = lambda t, n: torch.nn.functional.pad(t.reshape(t.shape[0], cols[n][0], -1), (0, cols[n][2] - cols[n][1])).reshape(t.shape[0], -1)
    padr = lambda t, n: torch.nn.functional.pad(t.reshape(cols[n][0], cols[n][1], -1), (0, 0, 0, cols[n][2] - cols[n][1])).reshape(-1, t.shape[1])
    filt = torch.cat([padr(w[n], n) for n in cols]).t().contiguous().cuda()
    ring = torch.full((9, taps, filt.shape[1]), 3.0, device="cuda")
    freq = torch.tensor([r["base"] ** (-2 * i / rot) for i in range(rot // 2)], device="cuda")
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    batch_all = PagedBatch([(0, L) for L in LENS], seed=1)
    kc = torch.zeros(batch_all.num_blocks, G, 16, dk, dtype=dtype, device="cuda")
    for mode in (0, 1, 2):
        vc = torch.zeros(batch_all.num_blocks, G, 16, dv, dtype=dtype, device="cuda")
        got_q = [[] for _ in LENS]
        for batch, begins, args in Portions():
            T = args["T"]
            proj = torch.cat([torch.cat([pads(u[n][b][s:s + m], n) for n in cols], 1) for b, s, m in batch]).cuda().to(dtype)
            pos = torch.tensor([s + i for b, s, m in batch for i in range(m)], dtype=torch.int32, device="cuda")
            smap = torch.tensor([batch_all.slot(b, s + i) for b, s, m in batch for i in range(m)], dtype=torch.int32, device="cuda")
            q_out = torch.zeros(T, H * dk, dtype=dtype, device="cuda")
            vf = torch.zeros(T, up(G * Dv, 4), dtype=dtype, device="cuda")
            if mode == 2:
                vf[:, :G * Dv] = torch.cat([first[b][s:s + m] for b, s, m in batch]).cuda().to(dtype)
            extra = {}
            if rot:
                table = torch.zeros(T, rot, device="cuda")
                K.rope_table(pos, freq, table, 1.0)
                extra = dict(rope=table, rot_dims=rot)
            K.heads_prepare(proj=proj, k_cache=kc, v_cache=vc, positions=pos, slot_map=smap, H=H, G=G, D=D, Dv=Dv, dk_pad=dk, dv_pad=dv, ldp=proj.stride(0),
                            k_off=H * dk, v_off=(H + G) * dk, block_size=16, dtype=K.storage_type(dtype), eps=1e-5, q_out=q_out, ldq=H * dk, conv_w=filt,
                            conv_ring=ring, conv_cols=filt.shape[1], taps=taps, v_first=vf if mode else None, ld_vf=vf.stride(0), v_mode=mode, v_mix=lam, **extra, **args)
            for (b, s, m), lo in zip(batch, begins):
                got_q[b].append(q_out[lo:lo + m].reshape(m, H, dk)[..., :D].float().cpu())
                if mode == 1:
                    close(vf[lo:lo + m, :G * Dv], want["v"][b][s:s + m].reshape(m, -1), tol)
        for b, L in enumerate(LENS):
            close(torch.cat(got_q[b]), want["q"][b], tol)
            v = want["v"][b]
            if mode == 2:
                v = (1 - lam) * v + lam * first[b].double().reshape(L, G, Dv)
            rows = [batch_all.slot(b, i) for i in range(L)]
            close(torch.stack([kc[s // 16, :, s % 16, :D] for s in rows]), want["k"][b], tol)
            close(torch.stack([vc[s // 16, :, s % 16, :Dv] for s in rows]), v, tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv,taps", [(4, 2, 32, 32, 4), (3, 1, 24, 40, 3), (2, 2, 64, 64, 2), (4, 1, 128, 128, 4), (40, 40, 64, 48, 3), (1, 1, 256, 256, 2),
                                           (2, 1, 144, 272, 1), (5, 5, 9, 13, 6)])
def test_channel_delta_in_portions(dtype, H, G, D, Dv, taps):
    """Everything between the projections and the output projection, over prompts cut at all kinds of places. Decays are slow and keys
    come back, so that what was lost early is still missing late."""
    K, bf, eps = k(), torch.bfloat16, 1e-3
    dk, dv = up(D, 16), up(Dv, 16)
    cols = {"q": (G, D, dk), "k": (G, D, dk), "v": (H, Dv, dv)}
    u = {n: [randn(L, h * d, seed=10 * i + j, dtype=bf) for j, L in enumerate(LENS)] for i, (n, (h, d, _)) in enumerate(cols.items())}
    for x in u["k"]:
        if len(x) > 100:
            x[100:104] = x[:4]                                  # an early key once more, far away
    for x in u["q"]:
        if len(x) > 130:
            x[130:134] = x[4:8]
    w = {n: randn(h * d, taps, seed=50 + i, dtype=bf) for i, (n, (h, d, _)) in enumerate(cols.items())}
    beta = [randn(L, H, seed=60 + j, dtype=bf) for j, L in enumerate(LENS)]
    low = [randn(L, H * D, seed=70 + j) for j, L in enumerate(LENS)]
    gate = [randn(L, H * Dv, seed=75 + j) for j, L in enumerate(LENS)]
    a_log, dt, norm = randn(H, seed=1, scale=0.5), randn(H * D, seed=2) - 5.0, randn(Dv, seed=3)
    want = []
    for j, L in enumerate(LENS):
        act = {n: oracle.silu(oracle.causal_conv(u[n][j].double(), w[n].double())).reshape(L, h, d) for n, (h, d, _) in cols.items()}
        rep = lambda t: t.repeat_interleave(H // G, 1)
        step = torch.nn.functional.softplus(low[j].double() + dt.double()).reshape(L, H, D)
        g = torch.exp(-a_log.double().exp()[:, None] * step)
        o = oracle.delta_scan(rep(oracle.unit(act["q"])) * D ** -0.5, rep(oracle.unit(act["k"])), act["v"], g, torch.sigmoid(beta[j].double()))
        want.append(oracle.rms_norm(o, norm.double(), eps) * torch.sigmoid(gate[j].double()).reshape(L, H, Dv))
    pads = lambda t, h, n: torch.nn.functional.pad(t.reshape(t.shape[0], h, -1), (0, n - t.shape[1] // h)).reshape(t.shape[0], -1)
    padr = lambda t, n: torch.nn.functional.pad(t.reshape(cols[n][0], cols[n][1], -1), (0, 0, 0, cols[n][2] - cols[n][1])).reshape(-1, t.shape[1])
    filt = torch.cat([padr(w[n], n) for n in cols]).t().contiguous().cuda()
    ring, state = torch.full((9, taps, filt.shape[1]), 3.0, device="cuda"), torch.full((9, H, dk, dv), 2.0, device="cuda")
    const = dict(conv_w=filt, conv_ring=ring, conv_cols=filt.shape[1], taps=taps, decay_a=a_log.exp().cuda(), state=state,
                 dt_bias=torch.nn.functional.pad(dt.reshape(H, D), (0, dk - D)).contiguous().cuda(), norm=torch.nn.functional.pad(norm, (0, dv - Dv)).cuda())
    got, b_off = [[] for _ in LENS], filt.shape[1]
    const["records"] = torch.full((K.channel_delta_record_floats(sum(LENS), len(LENS), H, dk, dv),), float("nan"), device="cuda")
    for batch, begins, args in Portions():
        T = args["T"]
        cat = lambda f: torch.cat([f(b, slice(s, s + m)) for b, s, m in batch])
        proj = torch.cat([cat(lambda b, r: pads(u[n][b][r], cols[n][0], cols[n][2])) for n in cols] + [cat(lambda b, r: pads(beta[b][r], 1, up(H, 16)))], 1)
        proj = proj.cuda().to(dtype)
        lows = torch.cat([cat(lambda b, r: pads(low[b][r], H, dk)), cat(lambda b, r: pads(gate[b][r], H, dv))], 1).cuda()
        out = torch.zeros(T, H * dv, dtype=dtype, device="cuda")
        K.channel_delta(proj=proj, low=lows, out=out, H=H, G=G, D=D, Dv=Dv, dk=dk, dv=dv, ldp=proj.stride(0), k_off=G * dk, v_off=2 * G * dk, b_off=b_off,
                        ld_low=lows.stride(0), gate_off=H * dk, ldo=H * dv, o_head=dv, dtype=K.storage_type(dtype), q_scale=D ** -0.5, eps=eps, **const, **args)
        for (b, _, m), lo in zip(batch, begins):
            got[b].append(out[lo:lo + m].float().cpu().reshape(m, H, dv)[..., :Dv])
    for g, v in zip(got, want):
        close(torch.cat(g), v, 3e-5 if dtype == torch.float32 else 1e-2)
    K.check_status("channel delta")


def test_decay_is_per_channel_and_exact_over_many_tokens():
    """One write, then two thousand tokens that only decay it (keys orthogonal to it): what is left is the product of the decays."""
    K, L, D = k(), 2000, 32
    proj = torch.zeros(L, 3 * D + 16)
    proj[0, D:D + 2], proj[0, 2 * D:3 * D] = 5.0, 4.0              # the first key has two channels
    proj[1:, D + 9] = 5.0                                         # later ones another
    proj[:, 0], proj[:, 1] = 5.0, -0.5                            # queries weigh the two channels unequally
    proj[:, 3 * D] = 30.0                                         # step size 1
    low = torch.zeros(L, 2 * D)
    low[:, 0], low[:, 1] = -6.0, -8.0                             # two slow decays
    low[:, D:] = 30.0
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    out, silu = torch.zeros(L, D, device="cuda"), lambda z: oracle.silu(torch.tensor(z, dtype=torch.float64))
    records = torch.empty(K.channel_delta_record_floats(L, 1, 1, D, D), device="cuda")
    K.channel_delta(proj=proj.cuda(), low=low.cuda(), conv_w=torch.ones(1, 3 * D, device="cuda"), conv_ring=torch.zeros(1, 1, 3 * D, device="cuda"),
                    decay_a=torch.ones(1, device="cuda"), dt_bias=torch.zeros(1, D, device="cuda"), norm=torch.ones(D, device="cuda"),
                    state=torch.zeros(1, 1, D, D, device="cuda"), out=out, records=records, subsequence_begins=i32([0, L]), past_lens=i32([0]), slots=i32([0]), B=1, T=L, H=1, G=1, D=D,
                    Dv=D, dk=D, dv=D, ldp=proj.stride(0), k_off=D, v_off=2 * D, b_off=3 * D, ld_low=2 * D, gate_off=D, conv_cols=3 * D, taps=1, ldo=D, o_head=D,
                    max_q_len=L, dtype=K.DT_F32, q_scale=1.0, eps=1.0)
    dt = torch.nn.functional.softplus(torch.tensor([-6.0, -8.0], dtype=torch.float64))
    keys = oracle.unit(silu([5.0, 5.0]))
    queries = oracle.unit(silu([5.0, -0.5]))
    t = torch.arange(1, L, dtype=torch.float64)[:, None]
    S = torch.exp(-t * dt) * keys * silu(4.0)
    o = (S * queries).sum(-1)                                     # (the later keys' values are zero: they write nothing)
    close(out[1:, 0], o / torch.sqrt(o * o + 1.0), 2e-5)

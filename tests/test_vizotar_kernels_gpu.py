"""Each Vizotar mechanism alone: the CUDA kernel against the plain fp32 functions of oracle/vizotar_oracle.py, in both storage
formats where the kernel has both (bf16 serving, fp32 exact).  Inputs are built so that a fault shows: streams that differ, gates at
their caps, a memory whose denominator sits on its floor, decays that differ wildly between channels, slots left full by others."""
import importlib
import math

import pytest
import torch

from oracle import vizotar_oracle as Z

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTS = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def ops():
    return importlib.import_module("nano-vllm-candle_b200.ops")


def tol(dt):
    return dict(rtol=3e-5, atol=3e-5) if dt == torch.float32 else dict(rtol=2e-2, atol=2e-2)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def gen(seed):
    return torch.Generator().manual_seed(seed)


def run_steps(sched, lens, slot_of, step_fn):
    """Drives step_fn(names, counts, starts, cu, pos, slots) -> rows over a schedule of (name, count) steps; returns name -> rows."""
    at = {n: 0 for n in lens}
    got = {n: [] for n in lens}
    for step in sched:
        cu, pos = [0], []
        for n, c in step:
            pos += list(range(at[n], at[n] + c))
            cu.append(cu[-1] + c)
        o = step_fn([n for n, _ in step], [c for _, c in step], [at[n] for n, _ in step], cu, pos, [slot_of[n] for n, _ in step])
        for b, (n, c) in enumerate(step):
            got[n].append(o[cu[b]:cu[b + 1]])
            at[n] += c
    assert at == lens
    return {n: torch.cat(v) for n, v in got.items()}


SCHED = [[("a", 20), ("b", 1)], [("b", 1), ("a", 1), ("c", 33)], [("c", 1), ("b", 2), ("a", 2)], [("b", 1), ("a", 1)], [("a", 13)], [("c", 63)]]
LENS = {"a": 37, "b": 5, "c": 97}
SLOTS = {"a": 2, "b": 0, "c": 3}


# ------------------------------------------------------------------------------------------ several residual streams
@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 8, 13, 16])
@pytest.mark.parametrize("H", [40, 37, 1100])
def test_a_sublayer_is_closed_and_the_next_one_opened(ctx, ops, dt, n, H):
    g = gen(n * H)
    N, eps = 6, 1e-3
    X, y0, y1 = torch.randn(n, N, H, generator=g), torch.randn(N, H, generator=g) * 30, torch.randn(N, H, generator=g) * 0.02
    b0, w0, w1, nw = (1 + 0.3 * torch.randn(H, generator=g) for _ in range(4))
    mix, out_w, in_w = torch.randn(n, n, generator=g) * 0.5, torch.randn(n, generator=g), torch.randn(n, generator=g)
    d = {k: v.to(DEV) for k, v in dict(y0=y0, y1=y1, b0=b0, w0=w0, w1=w1, nw=nw, mix=mix, out_w=out_w, in_w=in_w).items()}
    Xd = X.permute(1, 0, 2).contiguous().to(DEV)             # rows of a token side by side
    # two outputs, normed over the width with a weight each (the first with a bias in front) and averaged
    y = 0.5 * (Z.rms_norm(y0 + b0, w0, eps) + Z.rms_norm(y1, w1, eps))
    want = Z.write_streams(X, mix, out_w, y)
    got = ops.streams_norm(ctx, Xd, n, d["y0"], d["b0"], d["w0"], 0.5, d["y1"], d["w1"], 0.5, d["mix"], d["out_w"], d["in_w"], d["nw"], eps,
                           dt, x_out=Xd)                    # in place
    assert torch.allclose(Xd.cpu().permute(1, 0, 2), want, rtol=1e-5, atol=1e-4)
    assert torch.allclose(got.float().cpu(), Z.rms_norm(Z.read_streams(want, in_w), nw, eps), **tol(dt))
    if n > 1:          # the matrix is indexed [from, to]; a kernel that mixed rows with columns, or read new streams, would be elsewhere
        assert (Z.write_streams(X, mix.T, out_w, y) - want).abs().max() > 0.1
    # one plain output with a bias, out of place
    X1 = want
    want = Z.write_streams(X1, mix, out_w, y1 + b0)
    Xn = torch.zeros_like(Xd)
    keep = Xd.clone()
    got = ops.streams_norm(ctx, Xd, n, d["y1"], d["b0"], mix=d["mix"], out_w=d["out_w"], in_w=d["in_w"], norm_w=d["nw"], eps=eps, out_dtype=dt,
                           x_out=Xn)
    assert torch.equal(Xd, keep) and torch.allclose(Xn.cpu().permute(1, 0, 2), want, rtol=1e-5, atol=2e-4)
    assert torch.allclose(got.float().cpu(), Z.rms_norm(Z.read_streams(want, in_w), nw, eps), **tol(dt))
    # the head: the plain sum of the streams behind the last update, normed, of gathered rows; nothing is written back
    rows = i32([4, 0, 5])
    got = ops.streams_norm(ctx, Xd, n, d["y1"], d["b0"], mix=d["mix"], out_w=d["out_w"], norm_w=d["nw"], eps=eps, out_dtype=dt, rows=rows)
    assert torch.allclose(got.float().cpu(), Z.rms_norm(want.sum(0), d["nw"].cpu(), eps)[rows.cpu().long()], **tol(dt))
    assert torch.equal(Xd, keep)
    # the plain sum itself
    got = ops.streams_norm(ctx, Xd, n)
    assert torch.allclose(got.cpu(), X1.sum(0), rtol=1e-5, atol=2e-4)


@pytest.mark.parametrize("n", [1, 3, 6])
def test_streams_that_all_start_as_the_embedding(ctx, ops, n):
    g = gen(n)
    N, H, eps = 5, 72, 1e-5
    e, y, nw = torch.randn(N, H, generator=g), torch.randn(N, H, generator=g), 1 + 0.2 * torch.randn(H, generator=g)
    mix, out_w, in_w = torch.randn(n, n, generator=g), torch.randn(n, generator=g), torch.randn(n, generator=g)
    X = torch.stack([e] * n)
    ed, md, od, idv, nd = (t.to(DEV) for t in (e, mix, out_w, in_w, nw))
    got = ops.streams_norm(ctx, ed, n, in_w=idv, norm_w=nd, eps=eps)
    assert torch.allclose(got.cpu(), Z.rms_norm(Z.read_streams(X, in_w), nw, eps), rtol=2e-5, atol=2e-5)
    Xn = torch.empty(N, n, H, device=DEV)
    ops.streams_norm(ctx, ed, n, y.to(DEV), mix=md, out_w=od, in_w=idv, norm_w=nd, eps=eps, x_out=Xn)
    assert torch.allclose(Xn.cpu().permute(1, 0, 2), Z.write_streams(X, mix, out_w, y), rtol=1e-5, atol=1e-5)


def test_every_norm_of_the_streams_keeps_eps_inside_the_root(ctx, ops):
    N, H, eps = 2, 48, 1e-2
    X = torch.full((N, 2, H), 1e-4, device=DEV)
    y = torch.full((N, H), 1e-4, device=DEV)
    one = torch.ones(H, device=DEV)
    eye, ow = torch.eye(2, device=DEV), torch.ones(2, device=DEV)
    got = ops.streams_norm(ctx, X, 2, y, None, one, 1.0, mix=eye, out_w=ow, norm_w=one, eps=eps).cpu()
    s = 2 * (1e-4 + 1e-4 / math.sqrt(1e-8 + eps))
    assert torch.allclose(got, torch.full((N, H), s / math.sqrt(s * s + eps)), rtol=1e-5, atol=0)


# ------------------------------------------------------------------------------------------ convolution, whole-projection norms, rotation
@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("H,G,d,vd,taps,rot,scaled,pad", [(4, 2, 16, 24, 3, 8, True, 8), (3, 3, 20, 8, 4, 20, False, 4), (6, 1, 14, 10, 2, 6, True, 5),
                                                           (2, 2, 64, 128, 1, 32, True, 0), (1, 1, 6, 6, 5, 0, False, 3)])
def test_bias_convolution_whole_norm_and_rotation(ctx, ops, dt, H, G, d, vd, taps, rot, scaled, pad):
    """Portions down to one and two tokens (shorter than the taps), slots that an earlier owner left full; the norm spans all heads at
    once; biases are inside the convolution (and its state), zeros stand in front of a sequence - not biases."""
    g = gen(30)
    qw, kw, vw = H * d, G * d, G * vd
    C, eps = qw + kw + vw, 1e-3
    bias, cw = torch.randn(C, generator=g), torch.randn(C, taps, generator=g) * taps ** -0.5
    qn, kn = 1 + 0.3 * torch.randn(qw, generator=g), 1 + 0.3 * torch.randn(kw, generator=g)
    rotation = {"dims": rot, "base": 5000.0}
    if scaled:
        rotation["scaling"] = {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 1.0}
    rows = {n: torch.randn(T, pad + C, generator=g) * 2 for n, T in LENS.items()}
    want = {}
    for n, T in LENS.items():
        u, _ = Z.short_conv(rows[n][:, pad:] + bias, cw, torch.zeros(taps - 1, C))
        pos = torch.arange(T)
        q = Z.rotary_half(Z.rms_norm(u[:, :qw], qn, eps).view(T, H, d), pos, rotation).reshape(T, qw)
        k = Z.rotary_half(Z.rms_norm(u[:, qw:qw + kw], kn, eps).view(T, G, d), pos, rotation).reshape(T, kw)
        want[n] = torch.cat([q, k, u[:, qw + kw:]], -1)
    table = ops.rotary_table_scaled(ctx, 5000.0, rot, rotation.get("scaling"), 128) if rot else None
    conv_state = torch.randn(4, max(taps - 1, 1), C, generator=g).to(DEV)
    keep = conv_state[1].clone()
    full_bias = torch.cat([torch.full((pad,), 99.0), bias]).to(DEV)
    dev = {k: v.to(DEV) for k, v in dict(qn=qn, kn=kn).items()}
    cwd = cw.T.contiguous().to(DEV)

    def step(names, counts, starts, cu, pos, slots):
        x = torch.cat([rows[n][s:s + c] for n, c, s in zip(names, counts, starts)]).to(DEV)
        N = x.shape[0]
        decode = all(c == 1 for c in counts)
        q = torch.empty(N, qw, dtype=dt, device=DEV)
        kc, vc = torch.zeros(N + 9, kw, dtype=dt, device=DEV), torch.zeros(N + 9, vw, dtype=dt, device=DEV)
        slot_map = torch.randperm(N + 9, generator=g)[:N]
        ops.qkv_conv_prep(ctx, x, pad, H, G, d, vd, q, kc, vc, full_bias, cwd, conv_state, i32(slots), None if decode else i32(cu), i32(pos), dev["qn"],
                          dev["kn"], eps, rot, True, table, slot_map.to(torch.int32).to(DEV))
        kc, vc = kc.float().cpu(), vc.float().cpu()
        untouched = [s for s in range(N + 9) if s not in slot_map.tolist()]
        assert float(kc[untouched].abs().max()) == 0.0
        return torch.cat([q.float().cpu(), kc[slot_map], vc[slot_map]], -1)

    got = run_steps(SCHED, LENS, SLOTS, step)
    for n in LENS:
        assert torch.allclose(got[n], want[n], **tol(dt)), n
    if taps > 1:
        assert torch.equal(conv_state[1], keep)          # a slot nobody owns is not touched


# ------------------------------------------------------------------------------------------ window attention with a sink
@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("H,G,d,vd,window", [(5, 1, 96, 80, 9), (6, 2, 32, 16, 33), (3, 3, 20, 28, 5), (2, 2, 128, 64, 16), (4, 2, 64, 128, 0)])
def test_window_attention_with_a_sink_over_a_mixed_batch(ctx, ops, dt, H, G, d, vd, window):
    g = gen(31)
    lens, qlens, bs = [70, 1, 33, 129, 16], [70, 1, 2, 40, 1], 16
    sink = torch.randn(H, generator=g) * 2 + 1.0
    order = torch.randperm(24, generator=g).tolist()
    kc, vc, tables, want, qs = torch.zeros(24 * bs, G * d), torch.zeros(24 * bs, G * vd), [], [], []
    for n, m in zip(lens, qlens):
        k, v, q = torch.randn(n, G, d, generator=g), torch.randn(n, G, vd, generator=g), torch.randn(m, H, d, generator=g)
        if dt == torch.bfloat16:
            k, v, q = (t.bfloat16().float() for t in (k, v, q))
        bl, order = order[:(n + bs - 1) // bs], order[(n + bs - 1) // bs:]
        for j in range(n):
            kc[bl[j // bs] * bs + j % bs], vc[bl[j // bs] * bs + j % bs] = k[j].reshape(-1), v[j].reshape(-1)
        tables.append(bl)
        vis = Z.window_mask(torch.arange(n - m, n), n, window or None)
        o = torch.zeros(m, H, vd)
        for h in range(H):
            o[:, h] = Z.softmax_with_sink(q[:, h] @ k[:, h // (H // G)].T * 0.3, vis, sink[h]) @ v[:, h // (H // G)]
        want.append(o.reshape(m, H * vd))
        qs.append(q.reshape(m, H * d))
    width = max(len(t) for t in tables)
    cu = [0]
    for m in qlens:
        cu.append(cu[-1] + m)
    got = ops.attn_paged_wide(ctx, torch.cat(qs).to(dt).to(DEV), kc.to(dt).to(DEV), vc.to(dt).to(DEV), i32([t + [-1] * (width - len(t)) for t in tables]),
                              i32(lens), i32(cu), max(qlens), bs, H, G, d, vd, 0.3, window, sink.to(DEV), None, 1.0)
    assert torch.allclose(got.float().cpu(), torch.cat(want), **tol(dt))


@pytest.mark.parametrize("bs", [16, 64])
@pytest.mark.parametrize("window", [1, 39, 64, 65, 128, 200, 1000])
def test_long_portions_over_a_window_on_the_tensor_memory_kernel(ctx, ops, bs, window):
    """Heads of 128 numbers on tcgen05: whole prompts, portions behind a prefix that ends inside a page, short portions beside long ones; one
    key of huge score just inside the window of a row and just outside that of the next."""
    g = gen(32)
    H, G, d, scale = 4, 2, 128, 128 ** -0.5
    lens, qlens = [300, 131, 517, 70], [300, 64, 260, 3]
    sink = torch.randn(H, generator=g) + 1.0
    nb = sum((n + bs - 1) // bs for n in lens) + 2
    order = torch.randperm(nb, generator=g).tolist()
    kc = torch.full((nb * bs, G * d), float("nan"))                  # rows nobody wrote may hold anything
    vc = kc.clone()
    tables, want, qs, moved = [], [], [], []
    for n, m in zip(lens, qlens):
        k, v, q = torch.randn(n, G, d, generator=g), torch.randn(n, G, d, generator=g), torch.randn(m, H, d, generator=g)
        edge = n - m // 2                                            # row at position edge: its window starts at edge - window + 1
        j = max(edge - window + 1, 0)
        q[edge - (n - m), :] = q[edge - (n - m), 0]
        k[j] = q[edge - (n - m), 0] * 2.0
        if edge + 1 < n:
            q[edge + 1 - (n - m), :] = q[edge - (n - m), 0]
        k, v, q = (t.bfloat16().float() for t in (k, v, q))
        bl, order = order[:(n + bs - 1) // bs], order[(n + bs - 1) // bs:]
        for t in range(n):
            kc[bl[t // bs] * bs + t % bs], vc[bl[t // bs] * bs + t % bs] = k[t].reshape(-1), v[t].reshape(-1)
        tables.append(bl)
        pos = torch.arange(n - m, n)
        o, wide = torch.zeros(m, H, d), torch.zeros(m, H, d)
        for h in range(H):
            s = q[:, h] @ k[:, h // (H // G)].T * scale
            o[:, h] = Z.softmax_with_sink(s, Z.window_mask(pos, n, window), sink[h]) @ v[:, h // (H // G)]
            wide[:, h] = Z.softmax_with_sink(s, Z.window_mask(pos, n, window + 1), sink[h]) @ v[:, h // (H // G)]
        if j > 0 and edge + 1 < n:
            moved.append((o - wide)[edge + 1 - (n - m)].abs().max())
        want.append(o.reshape(m, H * d))
        qs.append(q.reshape(m, H * d))
    assert all(x > 0.3 for x in moved)                               # a window one token too wide would show
    width = max(len(t) for t in tables)
    cu = [0]
    for m in qlens:
        cu.append(cu[-1] + m)
    got = ops.prefill_attn_window(ctx, torch.cat(qs).bfloat16().to(DEV), kc.bfloat16().to(DEV), vc.bfloat16().to(DEV),
                                  i32([t + [-1] * (width - len(t)) for t in tables]), i32(lens), i32(cu), max(qlens), bs, H, G, scale, window, sink.to(DEV))
    assert torch.allclose(got.float().cpu(), torch.cat(want), rtol=2e-2, atol=2e-2)


# ------------------------------------------------------------------------------------------ matrix memory
def memory_want(data, H, d, vd, cap, bi, bf):
    q, k, v, zi, zf = data
    T = q.shape[0]
    i = Z.gate_cap(zi + bi, cap)
    f = torch.nn.functional.logsigmoid(Z.gate_cap(zf + bf, cap))
    o, *_ = Z.matrix_memory(q.view(T, H, d) * d ** -0.5, k.view(T, H, d), v.view(T, H, vd), i, f, torch.zeros(H, d, vd), torch.zeros(H, d), torch.zeros(H))
    return o.reshape(T, H * vd)


@pytest.mark.parametrize("form", ["token by token", "32 tokens at a time"])
@pytest.mark.parametrize("H,d,vd,cap,gate", [(3, 16, 24, 15.0, 1.0), (2, 40, 64, 6.0, 3.0), (1, 8, 1, 2.0, 9.0), (2, 200, 72, 15.0, 2.0), (4, 7, 40, 15.0, 20.0),
                                             (1, 128, 128, 10.0, 1.0), (2, 300, 33, 8.0, 2.0)])
def test_matrix_memory_between_portions_and_slots(ctx, ops, H, d, vd, cap, gate, form):
    """gate: spread of the gate inputs; the wide ones sit at both caps, so the running maximum jumps, forgets and rises from token to
    token.  q, k and v are columns of wider rows, as in a fused projection."""
    g = gen(40)
    cols = 2 * H * d + H * vd + 2 * H + 4
    rows = {n: torch.randn(T, cols, generator=g) for n, T in LENS.items()}
    for r in rows.values():
        r[:, -2 * H - 4:-4] *= gate
    bi, bf = torch.randn(H, generator=g) - 1.0, torch.randn(H, generator=g) + 2.0

    def split(r):
        return (r[:, :H * d], r[:, H * d:2 * H * d], r[:, 2 * H * d:2 * H * d + H * vd], r[:, -2 * H - 4:-H - 4], r[:, -H - 4:-4])

    want = {n: memory_want(split(r), H, d, vd, cap, bi, bf) for n, r in rows.items()}
    sl = (vd + 31) // 32
    state, nm = torch.randn(4, H, d, vd, generator=g).to(DEV), torch.randn(4, H, sl, d + 1, generator=g).to(DEV)
    keep = (state[1].clone(), nm[1].clone())
    bid, bfd = bi.to(DEV), bf.to(DEV)

    def step(names, counts, starts, cu, pos, slots):
        x = torch.cat([rows[n][s:s + c] for n, c, s in zip(names, counts, starts)]).to(DEV)
        decode = all(c == 1 for c in counts)
        q, k, v, zi, zf = split(x)
        return ops.memory_scan(ctx, q, k, v, zi, zf, bid, bfd, cap, state, nm, i32(slots), None if decode else i32(cu), i32(pos), H, d, vd,
                               max_qlen=max(counts) if form != "token by token" else 1).cpu()

    got = run_steps(SCHED, LENS, SLOTS, step)
    for n in LENS:
        scale = want[n].abs().max()
        assert (got[n] - want[n]).abs().max() < 2e-4 * max(1.0, float(scale)), n
        err = ((got[n] - want[n]).norm(dim=-1) / want[n].norm(dim=-1)).max()
        assert err < 2e-3, (n, float(err))               # a token whose |n . q| nearly cancels amplifies rounding
    assert torch.equal(state[1], keep[0]) and torch.equal(nm[1], keep[1])


@pytest.mark.parametrize("max_qlen", [1, 90])
def test_the_memory_starts_from_a_maximum_of_zero(ctx, ops, max_qlen):
    """Input gates at -8 and forget gates near 1: m stays near 0, so exp(-m) = 1 is far above |n . q| and the outputs stay tiny; a
    running maximum that started at minus infinity would divide the first token's value by |k . q| instead."""
    H, d, vd, T, cap = 2, 16, 8, 90, 15.0
    g = gen(41)
    q, k, v = (torch.randn(T, H * w, generator=g) for w in (d, d, vd))
    zi, zf = torch.full((T, H), -9.0), torch.full((T, H), 9.0)
    zero = torch.zeros(H)
    want = memory_want((q, k, v, zi, zf), H, d, vd, cap, zero, zero)
    # the same memory entered with m = -inf: the first token's state is k v^T with full weight
    first = (k[0].view(H, d) * q[0].view(H, d)).sum(-1) * d ** -0.5
    other = torch.sign(first)[:, None] * v[0].view(H, vd)
    assert (other - want[0].view(H, vd)).abs().max() > 0.3
    state, nm = torch.full((1, H, d, vd), 5.0, device=DEV), torch.full((1, H, 1, d + 1), 5.0, device=DEV)
    got = ops.memory_scan(ctx, q.to(DEV), k.to(DEV), v.to(DEV), zi.to(DEV), zf.to(DEV), zero.to(DEV), zero.to(DEV), cap, state, nm, i32([0]),
                          i32([0, T]), i32(list(range(T))), H, d, vd, max_qlen=max_qlen).cpu()
    assert torch.allclose(got, want, rtol=1e-3, atol=1e-6)


@pytest.mark.parametrize("cuts", [[400], [1] * 5 + [2, 33, 64, 296], [360] + [1] * 40])
def test_the_memory_carries_an_early_token(ctx, ops, cuts):
    """One token writes with a strong input gate along an axis that only the last token reads."""
    H, d, vd, cap = 2, 16, 8, 15.0
    T = sum(cuts)
    g = gen(42)
    q, k, v = torch.zeros(T, H, d), torch.zeros(T, H, d), torch.randn(T, H, vd, generator=g)
    k[:, :, 1] = 1.0
    k[3] = 0.0
    k[3, :, 0] = 1.0
    q[T - 1, :, 0] = 1.0
    zi, zf = torch.full((T, H), -3.0), torch.full((T, H), 6.0)
    zi[3] = 4.0
    zero = torch.zeros(H)
    want = memory_want((q.view(T, -1), k.view(T, -1), v.view(T, -1), zi, zf), H, d, vd, cap, zero, zero)[-1]
    assert want.abs().max() > 0.1
    state, nm = torch.full((1, H, d, vd), 7.0, device=DEV), torch.full((1, H, 1, d + 1), 7.0, device=DEV)
    at = 0
    for c in cuts:
        s = slice(at, at + c)
        o = ops.memory_scan(ctx, q[s].reshape(c, -1).to(DEV), k[s].reshape(c, -1).to(DEV), v[s].reshape(c, -1).to(DEV), zi[s].to(DEV), zf[s].to(DEV),
                            zero.to(DEV), zero.to(DEV), cap, state, nm, i32([0]), None if c == 1 else i32([0, c]), i32(list(range(at, at + c))), H, d, vd,
                            max_qlen=c)
        at += c
    assert torch.allclose(o.cpu()[-1], want, rtol=1e-3, atol=1e-5)


def test_a_long_run_of_closed_forget_gates_loses_no_digits(ctx, ops):
    """Forget gates at their lower cap (log -15 per token) for a whole chunk behind one open stretch: the running sum inside the chunk
    reaches -480; what a token sees of its neighbours still agrees with the token-by-token form."""
    H, d, vd, T, cap = 1, 32, 32, 64, 15.0
    g = gen(43)
    q, k, v = (torch.randn(T, H * w, generator=g) for w in (d, d, vd))
    zi, zf = torch.randn(T, H, generator=g) * 3, torch.full((T, H), -200.0)
    zf[::7] = 3.0
    zero = torch.zeros(H)
    want = memory_want((q, k, v, zi, zf), H, d, vd, cap, zero, zero)
    for max_qlen in (1, T):
        state, nm = torch.zeros(1, H, d, vd, device=DEV), torch.zeros(1, H, 1, d + 1, device=DEV)
        o = ops.memory_scan(ctx, q.to(DEV), k.to(DEV), v.to(DEV), zi.to(DEV), zf.to(DEV), zero.to(DEV), zero.to(DEV), cap, state, nm, i32([0]), i32([0, T]),
                            i32(list(range(T))), H, d, vd, max_qlen=max_qlen).cpu()
        err = (o - want).norm(dim=-1) / want.norm(dim=-1)
        assert err.max() < 2e-4, (max_qlen, float(err.max()))


# ------------------------------------------------------------------------------------------ delta rule with a decay per channel
def channel_want(x, p, H, G, d, vd, taps, qk, a):
    T = x.shape[0]
    z = {}
    for n, lo, hi in (("q", 0, qk), ("k", qk, 2 * qk), ("v", 2 * qk, 2 * qk + H * vd)):
        y, _ = Z.short_conv(x[:, lo:hi], p["conv"][lo:hi], torch.zeros(taps - 1, hi - lo))
        z[n] = torch.nn.functional.silu(y)
    q = Z.unit(z["q"].view(T, G, d)).repeat_interleave(H // G, 1) * d ** -0.5
    k = Z.unit(z["k"].view(T, G, d)).repeat_interleave(H // G, 1)
    beta = torch.sigmoid(x[:, 2 * qk + H * vd:2 * qk + H * vd + H])
    gg = torch.exp(-torch.exp(p["A_log"]).view(1, H, 1) * torch.nn.functional.softplus(a + p["dt_bias"]).view(T, H, d))
    o, _ = Z.channel_delta_rule(q, k, z["v"].view(T, H, vd), gg, beta, torch.zeros(H, d, vd))
    return o.reshape(T, H * vd)


@pytest.mark.parametrize("form", ["token by token", "32 tokens at a time"])
@pytest.mark.parametrize("H,G,d,vd,taps,spread", [(4, 2, 16, 24, 3, 1.0), (2, 2, 64, 48, 4, 3.0), (3, 1, 20, 7, 2, 6.0), (2, 1, 128, 128, 4, 2.0), (1, 1, 200, 40, 1, 2.0),
                                                  (2, 2, 6, 70, 5, 2.0), (1, 1, 300, 8, 2, 1.0)])
def test_channel_decays_between_portions_and_slots(ctx, ops, H, G, d, vd, taps, spread, form):
    """spread: how far the channels' decays lie apart (the wide ones range from nearly 1 to nothing within one token)."""
    g = gen(50)
    qk = G * d
    C = 2 * qk + H * vd
    p = {"conv": torch.randn(C, taps, generator=g) * taps ** -0.5, "A_log": torch.randn(H, generator=g) * 0.5,
         "dt_bias": torch.randn(H * d, generator=g) * spread - 1.0}
    rows = {n: torch.randn(T, C + H + 3, generator=g) for n, T in LENS.items()}
    acts = {n: torch.randn(T, H * d + 5, generator=g) for n, T in LENS.items()}
    want = {n: channel_want(rows[n], p, H, G, d, vd, taps, qk, acts[n][:, :H * d]) for n in LENS}
    state, conv_state = torch.randn(4, H, d, vd, generator=g).to(DEV), torch.randn(4, max(taps - 1, 1), C, generator=g).to(DEV)
    keep = (state[1].clone(), conv_state[1].clone())
    dev = {k: v.to(DEV) for k, v in p.items()}
    cw = p["conv"].T.contiguous().to(DEV)

    def step(names, counts, starts, cu, pos, slots):
        x, a = (torch.cat([src[n][s:s + c] for n, c, s in zip(names, counts, starts)]).to(DEV) for src in (rows, acts))
        decode = all(c == 1 for c in counts)
        o, *_ = ops.delta_rule(ctx, x, (0, qk, 2 * qk, C, 0), H, G, d, vd, taps, cw, conv_state, state, i32(slots), None if decode else i32(cu), i32(pos),
                               dev["A_log"], dev["dt_bias"], max_qlen=1 if form == "token by token" else max(counts), channel_a=a)
        return o.cpu()

    got = run_steps(SCHED, LENS, SLOTS, step)
    for n in LENS:
        assert torch.allclose(got[n], want[n], rtol=2e-4, atol=2e-5), (n, float((got[n] - want[n]).abs().max()))
    assert torch.equal(state[1], keep[0]) and (taps == 1 or torch.equal(conv_state[1], keep[1]))


def test_a_channel_decays_by_its_own_rate_and_no_other(ctx, ops):
    """Channel 0 keeps what it holds, channel 1 halves per token, channel 2 forgets at once: three keys, one per channel, written first and
    read at the end."""
    H, d, vd, T = 1, 8, 4, 40
    x = torch.zeros(T, 2 * d + vd + H)
    big = 40.0                                            # silu(big) = big; unit vectors need one large number
    for t in range(3):
        x[t, d + t] = big
        x[t, 2 * d:2 * d + vd] = torch.tensor([1.0, 2.0, 3.0, 4.0]) * (t + 1)
    x[3:, d + 7] = big                                    # later tokens write along another axis
    x[T - 1, 0:3] = big                                   # the last one reads channels 0, 1 and 2
    x[:, -1] = 30.0                                       # beta = 1
    a = torch.zeros(T, d)
    p = {"conv": torch.ones(2 * d + vd, 1), "A_log": torch.zeros(1), "dt_bias": torch.full((d,), -40.0)}
    p["dt_bias"][1] = math.log(math.e ** math.log(2.0) - 1.0)         # softplus = log 2
    p["dt_bias"][2] = 300.0
    want = channel_want(x, p, H, 1, d, vd, 1, d, a)
    v0 = torch.nn.functional.silu(torch.tensor([1.0, 2.0, 3.0, 4.0]))
    exact = (v0 + torch.nn.functional.silu(2 * torch.tensor([1.0, 2.0, 3.0, 4.0])) * 2.0 ** -(T - 2)) * 3 ** -0.5 * d ** -0.5
    assert torch.allclose(want[-1], exact, rtol=1e-4, atol=1e-5)
    for max_qlen in (1, T):
        o, *_ = ops.delta_rule(ctx, x.to(DEV), (0, d, 2 * d, 2 * d + vd, 0), H, 1, d, vd, 1, p["conv"].T.contiguous().to(DEV), torch.zeros(1, 1, 2 * d + vd, device=DEV),
                               torch.full((1, H, d, vd), 9.0, device=DEV), i32([0]), i32([0, T]), i32(list(range(T))), p["A_log"].to(DEV), p["dt_bias"].to(DEV),
                               max_qlen=max_qlen, channel_a=a.to(DEV))
        assert torch.isfinite(o).all() and torch.allclose(o.cpu(), want, rtol=1e-4, atol=1e-5)


# ------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("E,top", [(5, 2), (12, 2), (1, 1), (3, 3), (40, 4), (256, 8)])
def test_router_by_biased_logits_with_a_softmax_over_the_chosen(ctx, ops, E, top):
    g = gen(60)
    z, b = torch.randn(50, E + 3, generator=g) * 3, torch.randn(E, generator=g) * 2
    z[0] *= 40.0                                          # scores whose exponentials would overflow without the maximum
    idx, w = ops.moe_route_logits_ex(ctx, z.to(DEV), b.to(DEV), E, top, 1.0, ops.ROUTE_CHOSEN, True)
    v, wi = torch.topk(z[:, :E] + b, top, dim=-1)
    assert torch.equal(idx.cpu().long(), wi)
    assert torch.allclose(w.cpu(), torch.softmax(v, -1), rtol=1e-5, atol=1e-7)
    if 1 < top < E:                                       # neither a softmax over all experts nor weights without the bias
        assert (torch.gather(torch.softmax(z[:, :E] + b, -1), 1, wi) - torch.softmax(v, -1)).abs().max() > 0.05
        assert (torch.softmax(torch.gather(z[:, :E], 1, wi), -1) - torch.softmax(v, -1)).abs().max() > 0.05


@pytest.mark.parametrize("M", [1, 5, 64, 130, 700])
@pytest.mark.parametrize("ff,W,limit", [(64, 64, 0.6), (192, 128, 7.0), (1024, 512, 1.0), (64, 64, 0.0)])
def test_clamped_gated_unit_in_the_epilogue_of_a_product(ctx, ops, M, ff, W, limit):
    g = gen(61)
    h, wg, wu = (torch.randn(*s, generator=g).bfloat16() for s in ((M, W), (ff, W), (ff, W)))
    wg, wu = (wg * 2 * W ** -0.5).bfloat16(), (wu * 2 * W ** -0.5).bfloat16()
    gate, up = torch.clamp(h.float() @ wg.float().T, max=limit), torch.clamp(h.float() @ wu.float().T, -limit, limit)
    want = gate * torch.sigmoid(1.702 * gate) * (up + 1.0)
    got = ops.gemm_glu_clamp_mul(ctx, h.to(DEV), wg.to(DEV), wu.to(DEV), limit).float().cpu()
    assert torch.allclose(got, want, rtol=1e-2, atol=1e-2)

"""Each Buzutar mechanism alone: the CUDA kernel against plain fp32 code (oracle/buzutar_oracle.py and the function below), in both
storage formats (bf16 serving, fp32 exact).  Attention runs in every form the framework has for it: FMA, mma.sync (decode rows, short and
long portions, keys split over a cluster), tcgen05."""
import importlib
import math

import pytest
import torch

from oracle import buzutar_oracle as Z

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


# ------------------------------------------------------------------------------------------ norms behind the sublayers, logit cap
@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("H", [24, 37, 200, 1100, 5000])
def test_norm_behind_a_sublayer_and_the_plain_stream(ctx, ops, dt, H):
    """s = res + norm(y) w (plain weights); the next sublayer reads s itself in the storage format."""
    l = ctx.l
    g = torch.Generator().manual_seed(2)
    N, eps = 7, 1e-3
    res, y, wy = torch.randn(N, H, generator=g) * 3, torch.randn(N, H, generator=g) * 40, 1 + 0.3 * torch.randn(H, generator=g)
    d = [t.to(DEV) for t in (res, y, wy)]
    out = torch.full((N, H + 4), 9.0, dtype=dt, device=DEV)
    ro = torch.empty_like(d[0])
    P = ops._ptr
    f = 0 if dt == torch.bfloat16 else 1
    s = res + Z.rms_norm(y, wy, eps)
    assert l.nvc_rms_norm_sandwich(ctx.h, P(d[0]), P(d[1]), P(d[2]), P(ro), H, None, P(out), f, H + 4, eps, 0.0, None, N, H, ops._stream()) == 0
    assert torch.allclose(ro.cpu(), s, rtol=1e-5, atol=1e-5)
    assert torch.equal(out[:, :H].cpu(), ro.cpu().to(dt)) and (out[:, H:] == 9.0).all()
    # nothing pending: the stream and its copy
    assert l.nvc_rms_norm_sandwich(ctx.h, P(d[0]), None, None, P(ro), H, None, P(out), f, H + 4, eps, 0.0, None, N, H, ops._stream()) == 0
    assert torch.equal(ro.cpu(), res) and torch.equal(out[:, :H].cpu(), res.to(dt))


@pytest.mark.parametrize("V,ld", [(200, 256), (203, 203), (4097, 4160), (1, 5)])
def test_logits_are_capped_in_place(ctx, ops, V, ld):
    x = torch.randn(5, ld, generator=torch.Generator().manual_seed(1)) * 40
    d = x.to(DEV)
    ops.softcap_f32(ctx, d[:, :V], 17.0)
    assert torch.allclose(d[:, :V].cpu(), 17.0 * torch.tanh(x[:, :V] / 17.0), rtol=1e-5, atol=1e-5)
    assert torch.equal(d[:, V:].cpu(), x[:, V:])                 # padding columns stay


# ------------------------------------------------------------------------------------------ rotation
@pytest.mark.parametrize("dims,base,sc", [
    (32, 10000.0, {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}),
    (24, 777.5, {"factor": 1.5, "original": 300, "fast": 8.0, "slow": 0.5}),
    (16, 1e6, {"factor": 40.0, "original": 4096, "fast": 1.0, "slow": 1.0}),       # both bounds meet: the ramp is a step
    (8, 100.0, {"factor": 2.0, "original": 64, "fast": 1000.0, "slow": 0.001}),    # both bounds clamped
    (6, 50.0, {"factor": 1.0, "original": 64, "fast": 4.0, "slow": 1.0}),
    (10, 300.0, None),
])
def test_scaled_rotary_table(ctx, ops, dims, base, sc):
    got = ops.rotary_table_scaled(ctx, base, dims, sc, 700).cpu()
    rot = {"dims": dims, "base": base, "scaling": sc}
    f, m = Z.rotary_frequencies(rot)
    a = torch.arange(700).double().view(-1, 1) * f.view(1, -1)
    assert torch.allclose(got[..., 0], (a.cos() * m).float(), atol=1e-6) and torch.allclose(got[..., 1], (a.sin() * m).float(), atol=1e-6)
    if sc and sc["factor"] > 1.0:
        assert m > 1.0
        plain = Z.rotary_frequencies({"dims": dims, "base": base})[0]
        assert (f <= plain + 1e-12).all() and (f < plain).any()


# ------------------------------------------------------------------------------------------ queries and shared rows of the sigmoid mixer
@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("H,G,d", [(4, 2, 16), (3, 1, 10), (5, 5, 7), (6, 2, 64), (16, 8, 128), (80, 8, 128)])
def test_queries_and_rows_of_shared_keys_and_values(ctx, ops, dt, H, G, d):
    """q_out . row * key_scale must be the score of the normed query and the normed key; the row itself is the projected key."""
    g = torch.Generator().manual_seed(3)
    N, eps, coef, every = 9, 1e-2, 0.7, 8
    qw, kw = H * d, G * d
    q_off, k_off = 4, 4 + qw + 4
    x = torch.randn(N, k_off + kw + 4, generator=g) * torch.tensor([0.01, 1, 3, 10, 1, 1, 2, 2, 5]).view(-1, 1)
    wq, wk = 1 + 0.3 * torch.randn(qw, generator=g), 1 + 0.3 * torch.randn(kw, generator=g)
    pos = torch.tensor([0, 6, 7, 8, 15, 16, 1000, 7, 3])
    slots = [4, 0, -1, 9, 2, 1, 7, 3, 11]
    cache = torch.full((12, kw + 4), 7.0, dtype=dt, device=DEV)
    ks = torch.full((12,), 7.0, device=DEV)
    rep = wk.view(G, d).repeat_interleave(H // G, 0).reshape(-1)
    q = ops.qk_norm_fold_store(ctx, x.to(DEV), q_off, qw, k_off, kw, (wq * rep).to(DEV), eps, i32(pos.tolist()), cache, ks, i32(slots), coef, every)
    xq, xk = x[:, q_off:q_off + qw], x[:, k_off:k_off + kw]
    temp = Z.q_temperature(pos, {"coef": coef, "every": every}).view(-1, 1)
    assert temp[0] == 1.0 and temp[1] == 1.0 and temp[2] > 1.0 and temp[3] == temp[2]          # the step lies at p + 1 = every
    want_q = Z.rms_norm(xq, wq, eps) * temp * rep
    assert torch.allclose(q.float().cpu(), want_q, **tol(dt))
    got, gk = cache.float().cpu(), ks.cpu()
    for n in range(N):
        if slots[n] >= 0:
            assert torch.equal(got[slots[n], :kw], xk[n].to(dt).float())
            assert math.isclose(gk[slots[n]], 1.0 / math.sqrt(float((xk[n] ** 2).mean()) + eps), rel_tol=1e-5)
            s = (q.float().cpu()[n].view(G, H // G, d) * got[slots[n], :kw].view(G, 1, d)).sum(-1).reshape(-1) * gk[slots[n]]
            ref = ((Z.rms_norm(xq[n], wq, eps) * temp[n]).view(G, H // G, d) * Z.rms_norm(xk[n], wk, eps).view(G, 1, d)).sum(-1).reshape(-1)
            assert torch.allclose(s, ref, rtol=1e-4 if dt == torch.float32 else 2e-2, atol=(1e-4 if dt == torch.float32 else 3e-2) * d ** 0.5)
    untouched = [s for s in range(12) if s not in slots]
    assert (got[untouched] == 7.0).all() and (gk[untouched] == 7.0).all() and (got[:, kw:] == 7.0).all()


# ------------------------------------------------------------------------------------------ attention
def plain_attention(q, k, v, pos0, scale, window=0, sigmoid=False, bias=None, ks=None, sink=None, gate=None):
    """q: [T, H, d]; k: [n, G, d]; v: [n, G, vd]; the last T of n positions.  ks: [n] factors on the keys' scores."""
    T, H, _ = q.shape
    n, G, vd = v.shape
    vis = Z.window_mask(torch.arange(pos0, pos0 + T), n, window or None)
    out = torch.zeros(T, H, vd)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        if ks is not None:
            s = s * ks.view(1, -1)
        if sigmoid:
            p = torch.where(vis, torch.sigmoid(s + (bias[h] if bias is not None else 0.0)), torch.zeros(()))
        else:
            s = s.masked_fill(~vis, float("-inf"))
            if sink is not None:
                s = torch.cat([s, sink[h].expand(T, 1)], 1)
            p = torch.softmax(s, -1)[:, :n]
        out[:, h] = p @ v[:, g]
    out = out.reshape(T, H * vd)
    return out if gate is None else out * torch.sigmoid(gate)


class Batch:
    """Requests of different lengths on shuffled pages of one pool whose unused rows hold NaN; the last qlens[b] tokens of each are
    queries.  shared: the values are the leading vd numbers of the key rows."""

    def __init__(self, H, G, d, vd, lens, qlens, bs, dt, seed, shared, scaled, sigmoid, gate=False, boost=None, pb=-3.0):
        g = torch.Generator().manual_seed(seed)
        r = lambda *s: torch.randn(*s, generator=g).to(dt).float()
        self.H, self.G, self.d, self.vd, self.lens, self.qlens, self.bs, self.dt = H, G, d, vd, lens, qlens, bs, dt
        self.k = [r(n, G, d) for n in lens]
        self.v = [k[..., :vd] if shared else r(k.shape[0], G, vd) for k in self.k]
        self.q = [r(t, H, d) for t in qlens]
        self.ks = [0.5 + torch.rand(n, generator=g) for n in lens] if scaled else [None] * len(lens)
        self.bias = pb + torch.randn(H, generator=g) if sigmoid else None
        self.gate = [torch.randn(t, H * vd, generator=g) for t in qlens] if gate else [None] * len(lens)
        self.sigmoid, self.shared = sigmoid, shared
        if boost:                   # one key that every head of one query row scores high
            b, row, key, target = boost
            self.k[b][key] = (torch.randn(d, generator=g).expand(G, d) / 1.0).to(dt).float()
            if shared:
                self.v[b] = self.k[b][..., :vd]
            kk = self.k[b][key, 0]
            f = 1.0 if self.ks[b] is None else float(self.ks[b][key])
            self.q[b][row] = (kk * (target / (float(kk @ kk) * f))).to(dt).float()
        blocks = [-(-n // bs) for n in lens]
        perm = torch.randperm(sum(blocks) + 2, generator=g).tolist()
        nslots = (sum(blocks) + 2) * bs
        self.table, at = [], 0
        kc, vc, sc = torch.full((nslots, G * d), float("nan")), torch.full((nslots, G * vd), float("nan")), torch.full((nslots,), float("nan"))
        for b, n in enumerate(lens):
            pages = perm[at:at + blocks[b]]
            at += blocks[b]
            self.table.append(pages + [-1] * (max(blocks) - blocks[b]))
            slots = torch.tensor([pages[t // bs] * bs + t % bs for t in range(n)])
            kc[slots] = self.k[b].reshape(n, -1)
            vc[slots] = self.v[b].reshape(n, -1)
            if scaled:
                sc[slots] = self.ks[b]
        self.kc = kc.to(dt).to(DEV)
        self.vc = self.kc if shared else vc.to(dt).to(DEV)
        self.sc = sc.to(DEV) if scaled else None
        self.cu = [0]
        for t in qlens:
            self.cu.append(self.cu[-1] + t)

    def want(self, scale, window=0, sink=None):
        return torch.cat([plain_attention(self.q[b], self.k[b], self.v[b], n - self.qlens[b], scale, window, self.sigmoid, self.bias, self.ks[b], sink,
                                          self.gate[b]) for b, n in enumerate(self.lens)])

    def dev_q(self):
        return torch.cat(self.q).reshape(self.cu[-1], -1).to(self.dt).to(DEV)

    def dev_gate(self):
        return torch.cat(self.gate).to(DEV) if self.gate[0] is not None else None

    def wide(self, ctx, ops, scale, window=0, sink=None):
        decode = all(t == 1 for t in self.qlens)
        return ops.attn_paged_wide(ctx, self.dev_q(), self.kc, self.vc, i32(self.table), i32(self.lens), None if decode else i32(self.cu), max(self.qlens),
                                   self.bs, self.H, self.G, self.d, self.vd, scale, window, sink.to(DEV) if sink is not None else None, self.dev_gate(), 1.0,
                                   sigmoid=self.sigmoid, bias=self.bias.to(DEV) if self.sigmoid else None, key_scale=self.sc).float().cpu()

    def tcgen05(self, ctx, ops, scale, window=0, sink=None):
        return ops.prefill_attn_shared(ctx, self.dev_q(), self.kc, i32(self.table), i32(self.lens), i32(self.cu), max(self.qlens), self.bs, self.H, self.G,
                                       scale, window, sink.to(DEV) if sink is not None else None, self.sigmoid,
                                       self.bias.to(DEV) if self.sigmoid else None, self.sc, self.dev_gate()).float().cpu()


def close(got, want, dt):
    """Sigmoid weights are not normalised: outputs grow with the number of keys, so the bound is relative to a row's own size."""
    if dt == torch.float32:
        return torch.allclose(got, want, rtol=3e-5, atol=3e-5 * max(1.0, float(want.abs().max())))
    return bool(((got - want).abs() <= 2e-2 * want.abs() + 8e-3 * want.abs().amax(-1, keepdim=True).clamp_min(0.5)).all())


MIXED = dict(lens=[70, 1, 33, 129, 16], qlens=[70, 1, 2, 40, 1])
DECODE = dict(lens=[300, 1, 64, 65, 17, 40, 41], qlens=[1] * 7)
SIG_SHAPES = [(4, 2, 32), (3, 3, 40), (6, 1, 16), (6, 2, 64), (8, 2, 128), (5, 1, 96), (2, 2, 10)]


@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("H,G,d", SIG_SHAPES)
@pytest.mark.parametrize("batch", [MIXED, DECODE])
@pytest.mark.parametrize("bs", [16, 24, 64])
def test_sigmoid_attention_over_shared_rows(ctx, ops, dt, H, G, d, batch, bs):
    b = Batch(H, G, d, d, bs=bs, dt=dt, seed=H * d, shared=True, scaled=True, sigmoid=True, gate=True, **batch)
    assert close(b.wide(ctx, ops, 0.3), b.want(0.3), dt)


@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("batch", [MIXED, DECODE])
@pytest.mark.parametrize("window", [0, 9])
def test_sigmoid_attention_with_separate_values_and_no_factors(ctx, ops, dt, batch, window):
    b = Batch(4, 2, 48, 80, bs=16, dt=dt, seed=1, shared=False, scaled=False, sigmoid=True, **batch)
    assert close(b.wide(ctx, ops, 0.2, window), b.want(0.2, window), dt)


@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("batch", [MIXED, DECODE])
@pytest.mark.parametrize("G,d,vd,window", [(1, 48, 32, 1), (1, 48, 32, 16), (1, 128, 96, 17), (1, 40, 30, 5), (2, 64, 64, 33), (1, 128, 48, 0)])
def test_windowed_softmax_over_shared_rows(ctx, ops, dt, batch, G, d, vd, window):
    b = Batch(6, G, d, vd, bs=16, dt=dt, seed=d + window, shared=True, scaled=d == 64, sigmoid=False, **batch)
    assert close(b.wide(ctx, ops, 0.25, window), b.want(0.25, window), dt)


@pytest.mark.parametrize("H,G,d,vd,sigmoid", [(16, 1, 128, 96, False), (20, 1, 64, 48, False), (7, 1, 128, 128, False), (40, 2, 64, 64, True),
                                                (16, 1, 128, 128, True), (9, 3, 64, 64, True), (32, 4, 128, 128, True)])
@pytest.mark.parametrize("bs,window", [(16, 0), (64, 0), (48, 37), (64, 16), (16, 1)])
def test_decode_rows_in_the_transposed_form(ctx, ops, H, G, d, vd, sigmoid, bs, window):
    """Key rows of 64 and 128 numbers, up to 8, up to 16 and more query heads per key head (one or two n-tiles, several CTAs per key head)."""
    b = Batch(H, G, d, vd, lens=[300, 1, 64, 65, 17, 40, 41, 16, 530], qlens=[1] * 9, bs=bs, dt=torch.bfloat16, seed=H + window, shared=True,
              scaled=sigmoid, sigmoid=sigmoid, gate=sigmoid)
    assert close(b.wide(ctx, ops, 0.15, window), b.want(0.15, window), torch.bfloat16)
    if not sigmoid:
        sink = torch.linspace(-2, 4, H)
        assert close(b.wide(ctx, ops, 0.15, window, sink), b.want(0.15, window, sink), torch.bfloat16)


@pytest.mark.parametrize("sigmoid,window", [(True, 0), (False, 0), (False, 600), (True, 600)])
@pytest.mark.parametrize("lens", [[2100], [2047, 3], [1, 1500, 700]])
def test_decode_keys_split_over_a_cluster(ctx, ops, sigmoid, window, lens):
    """Few sequences with many keys: the CTAs of a cluster share a sequence's keys and merge their partial results."""
    b = Batch(8, 1, 128, 96 if not sigmoid else 128, lens=lens, qlens=[1] * len(lens), bs=64, dt=torch.bfloat16, seed=5, shared=True, scaled=sigmoid,
              sigmoid=sigmoid, gate=sigmoid, pb=-5.0)
    assert close(b.wide(ctx, ops, 0.1, window), b.want(0.1, window), torch.bfloat16)
    sink = None if sigmoid else torch.linspace(-1, 3, 8)
    if sink is not None:
        assert close(b.wide(ctx, ops, 0.1, window, sink), b.want(0.1, window, sink), torch.bfloat16)


@pytest.mark.parametrize("bs", [16, 32, 64, 128])
@pytest.mark.parametrize("batch", [
    dict(lens=[300, 64, 513, 129, 130], qlens=[300, 64, 200, 2, 129]),          # whole prompts, a prefix that ends inside a page, a two-token portion
    dict(lens=[1000], qlens=[999]),
    dict(lens=[128, 256], qlens=[128, 128]),
])
@pytest.mark.parametrize("sigmoid,G,H,window", [(True, 2, 4, 0), (True, 1, 3, 0), (True, 3, 3, 70), (False, 1, 5, 0), (False, 1, 6, 72), (False, 1, 2, 1),
                                                (False, 2, 4, 64), (False, 1, 3, 129)])
def test_tcgen05_portions_over_shared_rows(ctx, ops, bs, batch, sigmoid, G, H, window):
    b = Batch(H, G, 128, 128, bs=bs, dt=torch.bfloat16, seed=7 + window, shared=True, scaled=sigmoid, sigmoid=sigmoid, gate=sigmoid, pb=-4.0, **batch)
    got = b.tcgen05(ctx, ops, 0.09, window)
    assert close(got, b.want(0.09, window), torch.bfloat16)
    assert close(b.wide(ctx, ops, 0.09, window), b.want(0.09, window), torch.bfloat16)


def test_tcgen05_many_items_per_cta(ctx, ops):
    """More work items than resident CTAs: barriers and tensor memory are carried from item to item."""
    lens = [200 + 7 * i for i in range(40)]
    for sigmoid in (True, False):
        b = Batch(16, 8 if sigmoid else 1, 128, 128, lens=lens, qlens=lens, bs=64, dt=torch.bfloat16, seed=3, shared=True, scaled=sigmoid, sigmoid=sigmoid,
                  pb=-4.0)
        w = 0 if sigmoid else 100
        assert close(b.tcgen05(ctx, ops, 0.09, w), b.want(0.09, w), torch.bfloat16)


def test_tcgen05_sink_and_sigmoid_without_extras(ctx, ops):
    sink = torch.tensor([4.0, -2.0, 1.0])
    b = Batch(3, 1, 128, 128, lens=[200, 90], qlens=[150, 90], bs=64, dt=torch.bfloat16, seed=9, shared=True, scaled=False, sigmoid=False)
    for window in (0, 40):
        assert close(b.tcgen05(ctx, ops, 0.09, window, sink), b.want(0.09, window, sink), torch.bfloat16)
    b = Batch(4, 2, 128, 128, lens=[200, 90], qlens=[150, 90], bs=64, dt=torch.bfloat16, seed=9, shared=True, scaled=False, sigmoid=True)
    assert close(b.tcgen05(ctx, ops, 0.09), b.want(0.09), torch.bfloat16)


@pytest.mark.parametrize("form", ["fma", "mma", "mma_decode", "tcgen05"])
@pytest.mark.parametrize("n,key,seen", [
    (420, 419, True), (420, 420 - 72, True), (420, 420 - 73, False),              # itself, just inside and just outside the window
    (137, 137 - 72, True), (137, 64, False), (73, 1, True), (73, 0, False), (72, 0, True),
])
def test_the_windows_edge(ctx, ops, form, n, key, seen):
    """One key of huge score for the last row: inside the window it takes all the weight, one position further back none."""
    dt = torch.float32 if form == "fma" else torch.bfloat16
    b = Batch(2, 1, 128, 128, lens=[n], qlens=[1 if form == "mma_decode" else min(n, 70)], bs=16, dt=dt, seed=n + key, shared=True, scaled=False, sigmoid=False,
              boost=(0, -1, key, 60.0))
    got = (b.tcgen05 if form == "tcgen05" else b.wide)(ctx, ops, 1.0, 72)
    assert close(got, b.want(1.0, 72), dt)
    near = torch.allclose(got[-1].view(2, 128), b.k[0][key].expand(2, 128), rtol=3e-2, atol=3e-2)
    assert near == seen


@pytest.mark.parametrize("form", ["fma", "mma", "mma_decode", "tcgen05"])
@pytest.mark.parametrize("where", [0, 1, 15, 16, 17, 63, 64, 500, 1023, 1024])
def test_one_far_key_of_the_sigmoid_mixer(ctx, ops, form, where):
    """Biases near -7 leave every other key a weight of about a thousandth; one key with a score of 14 counts fully, wherever it lies."""
    dt = torch.float32 if form == "fma" else torch.bfloat16
    b = Batch(4, 2, 128, 128, lens=[1100], qlens=[1 if form == "mma_decode" else 130], bs=64, dt=dt, seed=where, shared=True, scaled=True, sigmoid=True, pb=-7.0,
              boost=(0, -1, where, 14.0))
    scale = 1.0
    b.q[0][:-1] *= 0.02                    # everyone else's scores stay near 0
    if form != "mma_decode":
        b.q[0][:-1] = b.q[0][:-1].to(dt).float()
    got = (b.tcgen05 if form == "tcgen05" else b.wide)(ctx, ops, scale)
    want = b.want(scale)
    assert close(got, want, dt)
    without = b.k[0][where].clone()
    assert float((got[-1].view(4, 128)[0] @ without[0]) / (without[0] @ without[0])) > 0.8       # its own value stands in the output


def test_small_sigmoid_weights_keep_their_relative_size(ctx, ops):
    """Weights of 2^-40 (a tanh form would round them to 0 or to 2^-12): a bias of -28 on every head."""
    for dt in DTS:
        b = Batch(4, 2, 128, 128, lens=[300], qlens=[130], bs=64, dt=dt, seed=2, shared=True, scaled=True, sigmoid=True, pb=-28.0)
        want = b.want(0.05)
        assert 0 < float(want.abs().max()) < 1e-8
        forms = [b.wide] if dt == torch.float32 else [b.wide, b.tcgen05]
        for f in forms:
            got = f(ctx, ops, 0.05)
            assert torch.allclose(got * 1e10, want * 1e10, rtol=2e-2, atol=float(want.abs().max()) * 1e8)

"""Buzutar through the runner and the engine: logits of every position against the plain fp32 oracle, whatever the schedule -
whole prompts, token-by-token decoding, portions down to two tokens, mixed batches, reused pages - plus greedy generation through
LLMEngine's own scheduler.  Small configurations whose sizes differ from one another (head counts, key / value / latent sizes, rotated
parts, windows around the block size, temperatures), layers without feed-forward, layers that read another layer's cache rows, models
that start with either mixer."""
import importlib

import numpy as np
import pytest
import torch

from oracle import buzutar_oracle as Z

pytestmark = pytest.mark.gpu
BLOCK = 16
YARN = {"factor": 6.0, "original": 48, "fast": 6.0, "slow": 0.5}


def cfg_a():
    """sigmoid / windowed latent / the same rows again with other heads and another window / sigmoid without feed-forward / latent."""
    return Z.make_config(vocab=200, width=96, layers=[
        Z.with_ff(Z.attention_cfg(6, 2, 16, scale=0.3, coef=0.6, every=16), 160),
        Z.with_ff(Z.latent_cfg(4, 16, 8, 24, 40, 48, scale=0.25, window=21, scaling=YARN), 96),
        Z.with_ff(Z.latent_cfg(3, 24, 8, 8, 40, 32, scale=0.2, window=9, scaling=YARN, kv_from=1), 64),
        Z.with_ff(Z.attention_cfg(4, 4, 24, scale=0.2, coef=0.3, every=5), None),
        Z.with_ff(Z.latent_cfg(5, 8, 16, 40, 24, 24, scale=0.3, window=16, base=500.0), 128),
    ])


def cfg_b():
    """Starts with a latent layer; sizes that are multiples of nothing; one head; no rotated part; a window of one token and one longer
    than any sequence; no window at all; a negative temperature coefficient; no temperature; no cap."""
    c = Z.make_config(vocab=203, width=100, eps=1e-3, embed_scale=1.0, cap=None, layers=[
        Z.with_ff(Z.latent_cfg(1, 20, 12, 28, 30, 25, scale=0.3, window=1, base=77.0, scaling={"factor": 2.5, "original": 20, "fast": 2.0, "slow": 1.0}), 72),
        Z.with_ff(Z.attention_cfg(5, 1, 10, scale=0.4, coef=-0.1, every=1), 33),
        Z.with_ff(Z.latent_cfg(5, 6, 0, 10, 17, 50, scale=0.4, window=5000), None),
        Z.with_ff(Z.latent_cfg(2, 12, 6, 12, 22, 16, scale=0.2, window=None), 40),
        Z.with_ff(Z.attention_cfg(1, 1, 36, scale=0.15), 56),
        Z.with_ff(Z.latent_cfg(7, 4, 6, 6, 22, 16, scale=0.5, window=17, kv_from=3), 24),
    ])
    c["layers"][4]["mixer"]["q_temp"] = None
    return c


def cfg_c():
    """Sizes of the tensor-pipe routes of the bf16 mode: cache rows of 64 and 128 numbers, sigmoid heads of 64 and 128 numbers (128-number
    rows take the tcgen05 kernel for long portions), windows shorter and longer than its tiles."""
    return Z.make_config(vocab=160, width=128, layers=[
        Z.with_ff(Z.latent_cfg(4, 32, 32, 32, 96, 64, scale=0.12, window=70, scaling=YARN), 192),
        Z.with_ff(Z.attention_cfg(4, 2, 128, scale=0.08, coef=0.4, every=32), 64),
        Z.with_ff(Z.latent_cfg(2, 64, 32, 64, 96, 32, scale=0.1, window=150, scaling=YARN, kv_from=0), None),
        Z.with_ff(Z.attention_cfg(6, 3, 64, scale=0.1, coef=0.2, every=100), 160),
        Z.with_ff(Z.latent_cfg(6, 16, 16, 16, 48, 64, scale=0.2, window=33), 64),
    ])


class Rig:
    def __init__(self, cfg, dtype, blocks=40, seed=0, chunked=True, seqs=4, weights=None):
        self.eng = importlib.import_module("nano-vllm-candle_b200.engine")
        self.cfg, self.dtype = cfg, dtype
        self.w = weights if weights is not None else Z.make_weights(cfg, seed)
        self.oracle = Z.Buzutar(cfg, self.w)
        self.ctx = self.eng.DeviceContext(0)
        T = blocks * BLOCK
        self.blocks = blocks
        self.runner = self.eng.ModelRunner.from_config(self.ctx, cfg, self.w.items(), num_kvcache_blocks=blocks, kvcache_block_size=BLOCK,
                                                       max_num_seqs=seqs, max_num_batched_tokens=T, max_model_len=T, dtype=dtype,
                                                       max_logit_rows=T)
        sc = self.eng.SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=T, eos=-1, num_kvcache_blocks=blocks,
                                      kvcache_block_size=BLOCK, enable_chunked_prefill=chunked, max_model_len=T)
        self.engine = self.eng.LLMEngine(self.eng.Scheduler(sc), self.runner, greedy=True)
        # error of a position: rms over the vocabulary of the mean-free logit difference, relative to the logits' own rms
        self.tol = 1e-4 if dtype == "float32" else 0.06

    def close(self):
        self.engine.close()
        self.runner.close()
        self.ctx.close()

    def want(self, tokens):
        return self.oracle.forward(tokens).numpy()

    def replay(self, prompts, schedule):
        """schedule: steps of [(request, count)]; every position's logits are collected; requests end when exhausted."""
        live, at = {}, {k: 0 for k in prompts}
        got = {k: np.zeros((len(v), self.cfg["vocab"]), np.float32) for k, v in prompts.items()}
        for step in schedule:
            entries = []
            for name, n in step:
                if name not in live:
                    live[name] = self.engine.open_request()
                entries.append((live[name], prompts[name][at[name]:at[name] + n], list(range(n))))
            lg = self.engine.step_forced(entries)
            row = 0
            for name, n in step:
                got[name][at[name]:at[name] + n] = lg[row:row + n]
                row += n
                at[name] += n
                if at[name] == len(prompts[name]):
                    self.engine.close_request(live.pop(name))
        assert all(at[k] == len(v) for k, v in prompts.items())
        return got

    def check(self, prompts, schedule):
        got = self.replay(prompts, schedule)
        for k, toks_ in prompts.items():
            err = self.rel_err(got[k], self.want(toks_))
            bad = err >= self.tol
            assert not bad.any(), \
                f"{k}: {int(bad.sum())} of {len(toks_)} positions over {self.tol}, first {int(np.argmax(bad))}, worst {err.max():.4g}"

    @staticmethod
    def rel_err(got, want):
        d = got - want
        d = d - d.mean(-1, keepdims=True)
        w = want - want.mean(-1, keepdims=True)
        return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean(-1))


def toks(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@pytest.fixture(scope="module", params=["float32", "bfloat16"])
def rig(request):
    r = Rig(cfg_a(), request.param)
    yield r
    r.close()


def test_whole_prompts_and_first_tokens(rig):
    V = rig.cfg["vocab"]
    rig.check({"one": toks(1, V, 1)}, [[("one", 1)]])
    rig.check({"two": toks(2, V, 2)}, [[("two", 2)]])
    rig.check({"three": toks(3, V, 2)}, [[("three", 3)]])
    rig.check({"p": toks(83, V, 2)}, [[("p", 83)]])
    rig.check({"page": toks(2 * BLOCK, V, 3)}, [[("page", 2 * BLOCK)]])


def test_residual_stream_after_every_layer(rig):
    p = toks(21, rig.cfg["vocab"], 4)
    tap = rig.runner.tap_residual(len(p))
    sid = rig.engine.open_request()
    rig.engine.step_forced([(sid, p, [0])])
    rig.engine.close_request(sid)
    res = []
    rig.oracle.forward(p, taps=res)
    assert tap.shape[0] == len(res) == 5
    for k, want in enumerate(res):
        assert np.abs(tap[k] - want.numpy()).max() < (2e-4 if rig.dtype == "float32" else 0.3), f"layer {k}"


def test_prefill_then_token_by_token(rig):
    p = toks(70, rig.cfg["vocab"], 5)
    rig.check({"d": p}, [[("d", 30)]] + [[("d", 1)]] * 40)
    rig.check({"d": p}, [[("d", 1)]] * 70)                       # decoding from the very first token, across page borders


def test_portions_of_many_sizes(rig):
    p = toks(121, rig.cfg["vocab"], 6)
    sizes = [2, 14, 16, 1, 17, 2, 31, 3, 33, 2]        # cuts before, at and after page borders
    assert sum(sizes) == 121
    rig.check({"c": p}, [[("c", n)] for n in sizes])
    rig.check({"c": p}, [[("c", 2)]] * 60 + [[("c", 1)]])
    rig.check({"c": p}, [[("c", 1)], [("c", 2)], [("c", 1)], [("c", 3)], [("c", 2)], [("c", 112)]])


def test_long_decoding(rig):
    p = toks(300, rig.cfg["vocab"], 7)
    rig.check({"l": p}, [[("l", 5)]] + [[("l", 1)]] * 295)


def test_mixed_batches_equal_each_request_alone(rig):
    V = rig.cfg["vocab"]
    pr = {"a": toks(90, V, 8), "b": toks(37, V, 9), "c": toks(3, V, 10), "d": toks(64, V, 11)}
    sched = [[("a", 40), ("b", 2)], [("a", 1), ("b", 20), ("c", 1)], [("a", 1), ("c", 1), ("d", 64)], [("a", 17), ("b", 1), ("c", 1)],
             [("a", 1), ("b", 14)]] + [[("a", 1)]] * 30
    assert all(sum(n for s in sched for k, n in s if k == name) == len(p) for name, p in pr.items())
    rig.check(pr, sched)


def test_a_request_left_out_of_steps_goes_on_later(rig):
    V = rig.cfg["vocab"]
    pr = {"a": toks(50, V, 12), "b": toks(45, V, 13)}
    rig.check(pr, [[("a", 10), ("b", 5)], [("b", 20)], [("b", 1)], [("a", 1), ("b", 1)], [("b", 18)], [("a", 39)]])


def test_steps_without_wanted_logits(rig):
    """Steps that ask for no logits: single tokens go through the captured decode step, portions through the mixed step; the next
    wanted position must not notice."""
    V = rig.cfg["vocab"]
    pa, pb = toks(60, V, 14), toks(45, V, 15)
    a, b = rig.engine.open_request(), rig.engine.open_request()
    rig.engine.step_forced([(a, pa[:20], []), (b, pb[:3], [])])
    for i in range(30):
        rig.engine.step_forced([(b, pb[3 + i:4 + i], []), (a, pa[20 + i:21 + i], [])])      # decode steps, nothing wanted
    rig.engine.step_forced([(a, pa[50:59], [])])
    lg = rig.engine.step_forced([(a, pa[59:], [0]), (b, pb[33:], [0, 11])])
    wa, wb = rig.want(pa), rig.want(pb)
    err = rig.rel_err(lg, np.stack([wa[59], wb[33], wb[44]]))
    assert err.max() < rig.tol, err
    rig.engine.close_request(a)
    rig.engine.close_request(b)


def test_pages_are_freed_and_used_again(rig):
    """The pool holds 40 pages; the requests below need 76 in total, at most 38 at a time."""
    V = rig.cfg["vocab"]
    free0 = rig.engine.num_free_blocks()
    for rnd in range(3):
        pr = {"x": toks(300, V, 20 + rnd), "y": toks(290, V, 30 + rnd)}
        rig.check(pr, [[("x", 150), ("y", 7)], [("x", 149), ("y", 282)], [("x", 1), ("y", 1)]])
        assert rig.engine.num_free_blocks() == free0
    # four live requests, closed in another order than opened
    for rnd in range(2):
        pr = {k: toks(20 + 3 * i, V, 40 + 10 * rnd + i) for i, k in enumerate("pqrs")}
        rig.check(pr, [[("p", 5), ("q", 23)], [("r", 10), ("p", 1), ("s", 2)], [("s", 27), ("p", 14), ("r", 16)]])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(dtype):
    r = Rig(cfg_b(), dtype, blocks=12, seed=3)
    try:
        V = r.cfg["vocab"]
        pr = {"a": toks(100, V, 1), "b": toks(19, V, 2)}
        r.check(pr, [[("a", 20), ("b", 19)], [("a", 2)], [("a", 27)], [("a", 1)]] + [[("a", 1)]] * 50)
    finally:
        r.close()


@pytest.mark.parametrize("dtype,flash", [("bfloat16", "1"), ("bfloat16", "0"), ("float32", "1")])
def test_sizes_of_the_tensor_pipe_routes(monkeypatch, dtype, flash):
    """Portions of 64 tokens and more - whole prompts, behind a cached prefix that ends inside a page, beside one-token sequences of
    the same step - with the tcgen05 attention route on and off: which kernel computed a position depends on the schedule, so both must
    agree with the oracle alike."""
    monkeypatch.setenv("NVC_BUZUTAR_FLASH", flash)
    r = Rig(cfg_c(), dtype, blocks=48, seed=12)
    try:
        V = r.cfg["vocab"]
        pr = {"a": toks(333, V, 60), "b": toks(131, V, 61), "c": toks(70, V, 62), "d": toks(5, V, 63)}
        sched = [[("a", 129), ("d", 1)], [("d", 1), ("a", 64), ("b", 77)], [("d", 1), ("a", 1), ("b", 3), ("c", 70)],
                 [("d", 1), ("b", 51), ("a", 139)], [("d", 1)]]
        assert all(sum(n for s in sched for k, n in s if k == name) == len(p) for name, p in pr.items())
        r.check(pr, sched)
        r.check({"w": toks(200, V, 64)}, [[("w", 200)]])
        r.check({"w": toks(200, V, 64)}, [[("w", 9)], [("w", 191)]])
        r.check({"w": toks(200, V, 64)}, [[("w", 150)]] + [[("w", 1)]] * 50)
    finally:
        r.close()


def sharp_latent_model(window, special=50, seed=30):
    """One latent layer in which head 0 scores the token `special` far above every other key, wherever it stands: the embedding gives
    that token alone a component along width 0 and every token the same component along width 1; latent 0 of the keys picks the first,
    latent 0 of the queries the second, and key / query number 0 of head 0 read them.  Random weights alone would average a single key away."""
    cfg = Z.make_config(vocab=60, width=64, embed_scale=1.0, cap=30.0, layers=[Z.with_ff(Z.latent_cfg(2, 16, 16, 16, 32, 32, scale=1.0, window=window), None)])
    w = Z.make_weights(cfg, seed)
    w["embed"][:, 0] = 0.0
    w["embed"][special, 0] = 8.0
    w["embed"][:, 1] = 4.0
    w["l0.mix.dkv"][0] = 0.0
    w["l0.mix.dkv"][0, 0] = 1.0
    w["l0.mix.dq"][0] = 0.0
    w["l0.mix.dq"][0, 1] = 1.0
    w["l0.mix.dq.norm"][0] = w["l0.mix.dkv.norm"][0] = 1.0
    w["l0.mix.uq"] *= 0.2
    w["l0.mix.uq"][0] = 0.0
    w["l0.mix.uq"][0, 0] = 1.0
    w["l0.mix.uk"][0] = 0.0
    w["l0.mix.uk"][0, 0] = 1.0
    return cfg, {k: v.bfloat16().float() for k, v in w.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,back,seen", [(37, 36, True), (37, 37, False), (16, 15, True), (16, 16, False), (200, 199, True), (200, 200, False)])
def test_a_key_at_the_edge_of_the_window(dtype, window, back, seen):
    """A token that occurs once, `back` positions before the end: with it just inside the window the last logits depend on it, one position
    further back they do not; whole prompt, portions cut around it, and decoding while the window passes over it."""
    cfg, w = sharp_latent_model(window)
    r = Rig(cfg, dtype, blocks=20, weights=w)
    try:
        n = 260
        p = [3 + (i * 7 % 11) for i in range(n)]
        p[n - 1 - back] = 50
        q = list(p)
        q[n - 1 - back] = 51
        moved = Rig.rel_err(r.want(p)[-1:], r.want(q)[-1:])[0]
        assert moved > 0.05 if seen else moved == 0.0
        scheds = [[[("w", n)]], [[("w", n - 1 - back)], [("w", 2)], [("w", back - 1)]], [[("w", n - back - 3)]] + [[("w", 1)]] * (back + 3)]
        for s in scheds:
            r.check({"w": p}, s)
        got_p, got_q = (r.replay({"w": t}, scheds[2])["w"][-1:] for t in (p, q))
        moved = Rig.rel_err(got_p, got_q)[0]
        assert moved > 0.05 if seen else moved < (1e-6 if dtype == "float32" else 1e-2)
    finally:
        r.close()


def sharp_sigmoid_model(seed=31, special=50):
    """One sigmoid layer whose keys all weigh next to nothing except the token `special`, which head 0 scores far above its bias: the
    embedding gives every token a component along width 1 (query number 0 reads it) and `special` one along width 0 (key number 0)."""
    cfg = Z.make_config(vocab=60, width=64, embed_scale=1.0, cap=30.0, layers=[Z.with_ff(Z.attention_cfg(2, 1, 16, scale=0.5, coef=0.3, every=100), None)])
    w = Z.make_weights(cfg, seed, pb=-7.0)
    w["embed"][:, 0] = 0.0
    w["embed"][special, 0] = 6.0
    w["embed"][:, 1] = 3.0
    w["l0.mix.q"] *= 0.2
    w["l0.mix.q"][0] = 0.0
    w["l0.mix.q"][0, 1] = 2.0
    w["l0.mix.k"][0] = 0.0
    w["l0.mix.k"][0, 0] = 1.0
    return cfg, {k: v.bfloat16().float() for k, v in w.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_far_back_among_hundreds(dtype):
    """A token that occurs once, 400 positions (25 pages) before the end: changing it moves the last logits, so it is attended to; the
    runner must agree with the oracle for a whole prompt, for portions and for decoding over it."""
    cfg, w = sharp_sigmoid_model()
    r = Rig(cfg, dtype, blocks=32, weights=w)
    try:
        n = 420
        p = [3 + (i * 7 % 11) for i in range(n)]
        p[n - 1 - 400] = 50
        q = list(p)
        q[n - 1 - 400] = 51
        assert Rig.rel_err(r.want(p)[-1:], r.want(q)[-1:])[0] > 0.1
        r.check({"w": p}, [[("w", n)]])
        r.check({"w": p}, [[("w", 13)], [("w", 200)], [("w", 2)], [("w", n - 215)]])
        r.check({"w": p}, [[("w", n - 20)]] + [[("w", 1)]] * 20)
        got_p, got_q = (r.replay({"w": t}, [[("w", n - 20)]] + [[("w", 1)]] * 20)["w"] for t in (p, q))
        assert Rig.rel_err(got_p[-1:], got_q[-1:])[0] > 0.1
    finally:
        r.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_temperature_steps_where_it_should(dtype):
    """A strong temperature that changes every eight positions: the oracle without it differs by far more than the tolerance from the
    first step on (position every - 1), and not at all before it."""
    cfg = Z.make_config(vocab=60, width=64, layers=[Z.with_ff(Z.attention_cfg(4, 2, 16, scale=0.5, coef=1.5, every=8), 64)])
    w = Z.make_weights(cfg, 6, pb=-1.0)
    r = Rig(cfg, dtype, blocks=8, weights=w)
    try:
        p = toks(70, 60, 3)
        flat = Z.make_config(vocab=60, width=64, layers=[Z.with_ff(Z.attention_cfg(4, 2, 16, scale=0.5, coef=0.0, every=8), 64)])
        moved = Rig.rel_err(Z.Buzutar(flat, w).forward(p).numpy(), r.want(p))
        assert moved[:7].max() == 0.0 and moved[7:].min() > 0.02
        r.check({"t": p}, [[("t", 70)]])
        r.check({"t": p}, [[("t", 7)]] + [[("t", 1)]] * 63)
    finally:
        r.close()


@pytest.mark.parametrize("dtype,chunked", [("float32", False), ("float32", True), ("bfloat16", True)])
def test_greedy_generation_through_the_scheduler(dtype, chunked):
    """LLMEngine.generate: the engine's own admission, paged prefill, graph-captured decode steps.  Every generated token must be the
    oracle's argmax on the same prefix (fp32) or within the bf16 error of its best logit."""
    r = Rig(cfg_a(), dtype, blocks=24, seed=5, chunked=chunked)
    try:
        V = r.cfg["vocab"]
        prompts = [toks(n, V, 50 + n) for n in (5, 33, 16, 2, 40, 9)]      # more requests than run at once
        outs = r.engine.generate(prompts, r.eng.SamplingParams(1.0, 12, True))
        assert len(outs) == 6
        for p, o in zip(prompts, outs):
            assert len(o.token_ids) == 12
            lg = r.want(p + o.token_ids[:-1])
            for i, t in enumerate(o.token_ids):
                row = lg[len(p) - 1 + i]
                assert row.max() - row[t] <= (2e-3 if dtype == "float32" else 0.6), f"token {i}"
        assert r.engine.num_free_blocks() == 24
    finally:
        r.close()


def test_prefix_caching():
    """The design keeps no state outside the paged rows: a second request with the same opening takes the first one's full blocks (rows
    and key factors alike) and must generate what it would alone."""
    r = Rig(cfg_a(), "float32", blocks=24, seed=5)
    try:
        sc = r.eng.SchedulerConfig(max_num_seqs=4, max_num_batched_tokens=24 * BLOCK, eos=-1, num_kvcache_blocks=24, kvcache_block_size=BLOCK,
                                   enable_prefix_caching=True, enable_chunked_prefill=True, max_model_len=24 * BLOCK)
        e = r.eng.LLMEngine(r.eng.Scheduler(sc), r.runner, greedy=True)
        V = r.cfg["vocab"]
        common = toks(3 * BLOCK + 5, V, 70)
        for tail in (toks(4, V, 71), toks(9, V, 72), toks(1, V, 73)):
            out = e.generate([common + tail], r.eng.SamplingParams(1.0, 8, True))[0]
            lg = r.want(common + tail + out.token_ids[:-1])
            for i, t in enumerate(out.token_ids):
                row = lg[len(common + tail) - 1 + i]
                assert row.max() - row[t] <= 2e-3
        e.close()
    finally:
        r.close()


def write_model_dir(path, cfg, weights):
    """config.json + model.safetensors (bf16) the way a checkpoint of this design is stored."""
    import json
    import struct
    header, blobs, at = {}, [], 0
    for name, t in weights.items():
        raw = t.bfloat16().contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
    (path / "config.json").write_text(json.dumps(cfg))


def test_command_line_tools_on_a_checkpoint_directory(tmp_path):
    """bin/trace_run and bin/generate: registry by config.json, native safetensors loader, the engine underneath."""
    import json
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = cfg_a()
    w = Z.make_weights(cfg, 9)
    oracle = Z.Buzutar(cfg, w)
    write_model_dir(tmp_path, cfg, w)
    V = cfg["vocab"]
    pa, pb = toks(41, V, 1), toks(9, V, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": pa[:30], "want": [0, 29]}, {"id": "b", "tokens": pb[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": pb[2:], "want": [6]}, {"id": "a", "tokens": pa[30:31], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": pa[31:], "want": [9]}, {"id": "b", "tokens": pb, "want": [8]}], "end": ["a", "b"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    la, lb = oracle.forward(pa).numpy(), oracle.forward(pb).numpy()
    want = {0: np.stack([la[0], la[29]]), 1: np.stack([lb[8], la[30]]), 2: np.stack([la[40], lb[8]])}
    for n, wv in want.items():
        got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, V)
        assert got.shape == wv.shape and Rig.rel_err(got, wv).max() < 1e-4, f"step {n}"
    g = subprocess.run([sys.executable, os.path.join(root, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32", "--prompt-ids",
                        ",".join(map(str, pb)) + ";" + ",".join(map(str, pa[:5])), "--max-tokens", "6", "--block-size", "16"],
                       capture_output=True, text=True, timeout=600)
    assert g.returncode == 0, g.stderr[-2000:]
    lines = [json.loads(ln) for ln in g.stdout.splitlines() if ln.startswith("{")]
    assert [ln["prompt"] for ln in lines] == [pb, pa[:5]]
    for ln in lines:
        lg = oracle.forward(ln["prompt"] + ln["tokens"][:-1]).numpy()
        for i, t in enumerate(ln["tokens"]):
            row = lg[len(ln["prompt"]) - 1 + i]
            assert row.max() - row[t] <= 2e-3

"""Plain fp32 restatement of the Vizotar design, one function per mechanism, slow on purpose.

Notation: W (width), V (vocab), T (new tokens of one sequence), pos0 (tokens before them).  Linear weights are
[out, in] and act as y = W x.  Instead of one residual stream there are n of them, X [n, T, W], all equal to
embed[token] at first.  A sublayer f (mixer or feed-forward, behind a plain RMS norm) reads a weighted sum of the
streams and every stream is rebuilt from all the old ones plus the sublayer's output:

    u = sum_s in_s X_s;   y = f(norm(u));   X_t <- sum_s mix[s, t] X_s + out_t y

The logits are the embedding table against the normed sum of the streams.  Mixers:

  parallel             two mixers that read the same h, their outputs RMS-normed over the width with a weight each
                       and averaged:
      window attention     grouped-query softmax attention; projections with biases, a short causal convolution over
                           time per channel of q, k and v, one RMS norm over the whole q (and k) projection,
                           rotate-half positions with YaRN frequencies, a sliding window, a learned sink
      matrix memory        mLSTM: per head S, n with exponential input gate and sigmoid forget gate in a
                           max-stabilised form (the running maximum starts at 0), per-head RMS norm, sigmoid gate
  channel_delta        gated delta rule with one decay per head AND key channel (a low-rank projection), short
                       convolutions with silu, unit q and k, low-rank sigmoid output gate

Feed-forward: dense clamped gated units, or experts chosen by biased router logits with a softmax over the chosen.

The caches are explicit: every function takes what earlier tokens left and returns what it leaves, so that the
same code serves whole prompts, portions and token-by-token decoding.  Everything here is float32 torch on the
CPU; nothing is shared with the CUDA path.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


# ------------------------------------------------------------------------------------------ streams

def read_streams(X: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """X: [n, T, W] -> what the sublayer reads, [T, W]."""
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + w_in[s] * X[s]
    return u


def write_streams(X: torch.Tensor, mix: torch.Tensor, w_out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """mix is indexed [from, to]; every new stream comes from the OLD ones."""
    new = []
    for t in range(X.shape[0]):
        z = w_out[t] * y
        for s in range(X.shape[0]):
            z = z + mix[s, t] * X[s]
        new.append(z)
    return torch.stack(new)


# ------------------------------------------------------------------------------------------ shared pieces

def short_conv(x: torch.Tensor, w: torch.Tensor, tail: torch.Tensor):
    """x: [T, C] new inputs, w: [C, taps], tail: [taps - 1, C] the inputs in front of them.  y_t = sum_j w[:, j] x_(t - taps + 1 + j);
    returns (y, the last taps - 1 inputs)."""
    taps = w.shape[1]
    z = torch.cat([tail, x], 0)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * z[t + j]
    return y, z[z.shape[0] - (taps - 1):].clone()


def yarn_ramp(dims: int, base: float, s: dict) -> torch.Tensor:
    """Per pair: 0 = the frequency stays, 1 = it is divided by the factor."""
    def pair_of(turns):          # the (fractional) pair that makes `turns` turns within the original length
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(s["fast"])), 0)
    hi = min(math.ceil(pair_of(s["slow"])), dims - 1)
    i = torch.arange(dims // 2, dtype=torch.float64)
    return ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)


def rotary_half(x: torch.Tensor, pos: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x: [T, heads, d]; pairs (i, i + dims / 2) of the first rot.dims numbers are turned, the rest passes."""
    if not rot or rot["dims"] == 0:
        return x
    dims, base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
    half = dims // 2
    f = torch.tensor(base, dtype=torch.float64) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    m = 1.0
    if s:
        ramp = yarn_ramp(dims, base, s)
        f = f / s["factor"] * ramp + f * (1.0 - ramp)
        m = 0.1 * math.log(s["factor"]) + 1.0
    a = pos.double().view(-1, 1) * f.view(1, -1)
    c, sn = (a.cos() * m).float()[:, None], (a.sin() * m).float()[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * sn, v * c + u * sn, x[..., dims:]], -1)


def window_mask(pos: torch.Tensor, keys: int, size: Optional[int]) -> torch.Tensor:
    """[T, keys]: a position sees itself and the size - 1 tokens before it (size None: every earlier token)."""
    back = pos.view(-1, 1) - torch.arange(keys).view(1, -1)
    return (back >= 0) & (back < size) if size else back >= 0


def softmax_with_sink(s: torch.Tensor, visible: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """s: [T, keys]; one more term exp(sink) in the denominator, which has no key and no value."""
    z = torch.cat([s.masked_fill(~visible, float("-inf")), sink.expand(s.shape[0], 1)], -1)
    return torch.softmax(z, -1)[:, :-1]


# ------------------------------------------------------------------------------------------ window attention (left)

def window_attention(h: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float, pos0: int, state: Optional[dict]):
    """state = {"K": [pos0, G, d], "V": [pos0, G, vd], "q" / "k" / "v": [taps - 1, channels]} of the tokens before (None: none)."""
    T, H, G, d, vd, taps = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    width = {"q": H * d, "k": G * d, "v": G * vd}
    if state is None:
        state = {"K": torch.zeros(0, G, d), "V": torch.zeros(0, G, vd), **{n: torch.zeros(taps - 1, c) for n, c in width.items()}}
    new, z = {}, {}
    for n in "qkv":
        z[n], new[n] = short_conv(h @ p[n].T + p[n + ".b"], p[n + ".conv"], state[n])
    pos = torch.arange(pos0, pos0 + T)
    q = rotary_half(rms_norm(z["q"], p["q.norm"], eps).view(T, H, d), pos, m.get("rot"))
    k = rotary_half(rms_norm(z["k"], p["k.norm"], eps).view(T, G, d), pos, m.get("rot"))
    new["K"] = torch.cat([state["K"], k], 0)
    new["V"] = torch.cat([state["V"], z["v"].view(T, G, vd)], 0)
    vis = window_mask(pos, pos0 + T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, vd)
    for hh in range(H):
        g = hh // (H // G)
        s = q[:, hh] @ new["K"][:, g].T * m["scale"]
        out[:, hh] = softmax_with_sink(s, vis, p["sink"][hh]) @ new["V"][:, g]
    return out.reshape(T, H * vd) @ p["o"].T + p["o.b"], new


# ------------------------------------------------------------------------------------------ matrix memory (right)

def gate_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def matrix_memory(q, k, v, i, f, S, n, m):
    """q, k: [T, H, d]; v: [T, H, vd]; i, f: [T, H] log gates; S [H, d, vd], n [H, d], m [H].  Returns (o [T, H, vd], S, n, m)."""
    T, H, _ = q.shape
    o = torch.zeros(T, H, v.shape[-1])
    S, n, m = S.clone(), n.clone(), m.clone()
    for t in range(T):
        for hh in range(H):
            mt = torch.maximum(f[t, hh] + m[hh], i[t, hh])
            keep, add = torch.exp(f[t, hh] + m[hh] - mt), torch.exp(i[t, hh] - mt)
            S[hh] = keep * S[hh] + add * torch.outer(k[t, hh], v[t, hh])
            n[hh] = keep * n[hh] + add * k[t, hh]
            m[hh] = mt
            o[t, hh] = (S[hh].T @ q[t, hh]) / (torch.maximum((n[hh] @ q[t, hh]).abs(), torch.exp(-mt)) + 1e-6)
    return o, S, n, m


def memory_mixer(h: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float, state: Optional[dict]):
    T, H, d, vd, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    if state is None:
        state = {"S": torch.zeros(H, d, vd), "n": torch.zeros(H, d), "m": torch.zeros(H)}
    q = (h @ p["q"].T).view(T, H, d) * d ** -0.5
    k = (h @ p["k"].T).view(T, H, d)
    v = (h @ p["v"].T).view(T, H, vd)
    i = gate_cap(h @ p["i"].T + p["i.b"], cap)
    f = torch.nn.functional.logsigmoid(gate_cap(h @ p["f"].T + p["f.b"], cap))
    o, S, n, mm = matrix_memory(q, k, v, i, f, state["S"], state["n"], state["m"])
    o = rms_norm(o, None, eps).reshape(T, H * vd) * p["norm"] * torch.sigmoid(h @ p["g"].T)
    return o @ p["o"].T, {"S": S, "n": n, "m": mm}


def parallel_mixer(h, p, m, eps, pos0, state: Optional[dict]):
    left, right = sub(p, "left."), sub(p, "right.")
    state = state or {}
    yl, sl = window_attention(h, left, m["left"], eps, pos0, state.get("left"))
    yr, sr = memory_mixer(h, right, m["right"], eps, state.get("right"))
    return 0.5 * (rms_norm(yl, left["out"], eps) + rms_norm(yr, right["out"], eps)), {"left": sl, "right": sr}


# ------------------------------------------------------------------------------------------ delta rule with channel decays

def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta_rule(q, k, v, g, beta, S):
    """q, k, g: [T, H, d] (g: decay of every row of S); v: [T, H, vd]; beta: [T, H]; S: [H, d, vd].  Returns (o [T, H, vd], S)."""
    T, H, _ = q.shape
    o = torch.zeros(T, H, v.shape[-1])
    S = S.clone()
    for t in range(T):
        for hh in range(H):
            Sh = S[hh] * g[t, hh][:, None]
            u = beta[t, hh] * (v[t, hh] - Sh.T @ k[t, hh])
            Sh = Sh + torch.outer(k[t, hh], u)
            o[t, hh] = Sh.T @ q[t, hh]
            S[hh] = Sh
    return o, S


def channel_delta_mixer(h: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float, state: Optional[dict]):
    T, H, G, d, vd, taps = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    if state is None:
        state = {"S": torch.zeros(H, d, vd), "q": torch.zeros(taps - 1, G * d), "k": torch.zeros(taps - 1, G * d),
                 "v": torch.zeros(taps - 1, H * vd)}
    new, z = {}, {}
    for n in "qkv":
        y, new[n] = short_conv(h @ p[n].T, p[n + ".conv"], state[n])
        z[n] = torch.nn.functional.silu(y)
    rep = H // G
    q = unit(z["q"].view(T, G, d)).repeat_interleave(rep, 1) * d ** -0.5
    k = unit(z["k"].view(T, G, d)).repeat_interleave(rep, 1)
    beta = torch.sigmoid(h @ p["b"].T)
    a = (h @ p["a1"].T) @ p["a2"].T + p["dt_bias"]
    g = torch.exp(-torch.exp(p["A_log"]).view(1, H, 1) * torch.nn.functional.softplus(a).view(T, H, d))
    o, new["S"] = channel_delta_rule(q, k, z["v"].view(T, H, vd), g, beta, state["S"])
    o = rms_norm(o, p["norm"], eps).reshape(T, H * vd) * torch.sigmoid((h @ p["g1"].T) @ p["g2"].T)
    return o @ p["o"].T, new


# ------------------------------------------------------------------------------------------ feed-forward

def dense_ff(h, p, limit: float):
    g = torch.clamp(h @ p["gate"].T, max=limit)
    u = torch.clamp(h @ p["up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ p["down"].T


def route(h, p, m):
    """The `top` experts with the largest biased logits; weights: softmax over the chosen logits.  (idx, weights) [T, top]."""
    z = h @ p["router"].T + p["router.b"]
    v, idx = torch.topk(z, m["router"]["top"], dim=-1)
    return idx, torch.softmax(v, -1)


def expert(h, p, e: int):
    return (torch.nn.functional.silu(h @ p[f"e{e}.gate"].T) * (h @ p[f"e{e}.up"].T)) @ p[f"e{e}.down"].T


def moe_ff(h, p, m):
    idx, wts = route(h, p, m)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            out[t] += wts[t, j] * expert(h[t: t + 1], p, int(idx[t, j]))[0]
    return out


def sub(params: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.float() for k, v in params.items() if k.startswith(prefix)}


class Vizotar:
    """The whole model over explicit per-request caches.  cfg: the dict of config.json; params: name -> tensor.  rows: a dtype that the
    rows in front of every sublayer are rounded to (None: not rounded) - how far rounding alone moves a position's logits; the first
    outputs of a recurrence are a sign, sign(k . q) v / rms(v), and some prompts sit close to the jump."""

    def __init__(self, cfg: dict, params: Dict[str, torch.Tensor], rows: Optional[torch.dtype] = None):
        self.cfg = cfg
        self.rows = rows
        self.p = {k: v.float() for k, v in params.items()}
        self.eps = cfg["norm"]["eps"]

    def owner(self, i: int) -> int:
        j = self.cfg["layers"][i].get("weights_of")
        return i if j is None else j

    def sublayer_row(self, X: torch.Tensor, w_in: torch.Tensor, norm: torch.Tensor) -> torch.Tensor:
        h = rms_norm(read_streams(X, w_in), norm, self.eps)
        return h if self.rows is None else h.to(self.rows).float()

    def new_cache(self) -> dict:
        return {"len": 0, "state": {}}

    def forward(self, tokens: List[int], cache: Optional[dict] = None, taps: Optional[list] = None) -> torch.Tensor:
        """Runs T new tokens of one request on top of `cache` (None: a whole prompt from an empty cache); returns logits [T, V]."""
        cfg, eps = self.cfg, self.eps
        if cache is None:
            cache = self.new_cache()
        pos0, state = cache["len"], cache["state"]
        e = self.p["embed"][torch.tensor(tokens)]
        X = torch.stack([e] * cfg["streams"])
        for i, ly in enumerate(cfg["layers"]):
            lp = sub(self.p, f"l{self.owner(i)}.")
            mp, m = sub(lp, "mix."), ly["mixer"]
            h = self.sublayer_row(X, lp["hc1.in"], lp["norm1"])
            if ly["type"] == "parallel":
                y, state[i] = parallel_mixer(h, mp, m, eps, pos0, state.get(i))
            elif ly["type"] == "channel_delta":
                y, state[i] = channel_delta_mixer(h, mp, m, eps, state.get(i))
            else:
                raise ValueError(ly["type"])
            X = write_streams(X, lp["hc1.mix"], lp["hc1.out"], y)
            if ly.get("mlp"):
                h = self.sublayer_row(X, lp["hc2.in"], lp["norm2"])
                fp = sub(lp, "mlp.")
                y = dense_ff(h, fp, ly["mlp"]["limit"]) if ly["mlp"]["kind"] == "dense" else moe_ff(h, fp, ly["mlp"])
                X = write_streams(X, lp["hc2.mix"], lp["hc2.out"], y)
            if taps is not None:
                taps.append(X.sum(0))
        cache["len"] = pos0 + len(tokens)
        return rms_norm(X.sum(0), self.p["final.norm"], eps) @ self.p["embed"].T


# ------------------------------------------------------------------------------------------ small configurations

def delta_cfg(heads=4, kv_heads=2, dim=24, vdim=20, conv=3) -> dict:
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def parallel_cfg(heads=6, kv_heads=2, dim=32, vdim=16, conv=4, window=11, rot_dims=16, base=10000.0, scaling=None, scale=0.2, mheads=3, mdim=20,
                 mvdim=28, cap=6.0) -> dict:
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale}
    if rot_dims is not None:
        left["rot"] = {"dims": rot_dims, "base": base}
        if scaling is not None:
            left["rot"]["scaling"] = dict(scaling)
    if window is not None:
        left["mask"] = {"size": window}
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": mheads, "dim": mdim, "vdim": mvdim, "gate_cap": cap}}}


def with_dense(layer: dict, ff: int = 72, limit: float = 0.8) -> dict:
    return {**layer, "mlp": {"kind": "dense", "ff": ff, "limit": limit}}


def with_moe(layer: dict, experts: int = 5, top: int = 2, ff: int = 40) -> dict:
    return {**layer, "mlp": {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}}


def with_none(layer: dict) -> dict:
    return {**layer, "mlp": None}


def again(layers: List[dict], j: int) -> dict:
    """One more run of layer j's weights, with a cache of its own."""
    return {**layers[j], "weights_of": j}


def make_config(vocab=200, width=96, layers=None, eps=1e-5, streams=2) -> dict:
    return {"architecture": "Vizotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers}


def make_weights(cfg: dict, seed: int = 0, bf16_values: bool = True, rank_a: int = 12, rank_g: int = 20, sink: float = 0.5) -> Dict[str, torch.Tensor]:
    """Random weights under the checkpoint's names; values bf16-representable by default so that the bf16 and fp32 paths load
    identical numbers.  rank_a / rank_g: the inner sizes of the low-rank decay and gate projections (a tensor's shape, not config).
    The recurrences' keys lean towards their queries: a first output is sign(k . q) v / rms(v), and independent keys and queries put
    some token of every prompt so close to the jump that bf16 rounding decides it."""
    gen = torch.Generator().manual_seed(seed)
    W, n = cfg["width"], cfg["streams"]

    def fix(t):
        return t.bfloat16().float() if bf16_values else t

    def rnd(*shape, s=1.0):
        return fix(torch.randn(*shape, generator=gen) * s)

    def one(k):
        return fix(1.0 + 0.2 * torch.randn(k, generator=gen))

    def lin(o, i):
        return rnd(o, i, s=i ** -0.5)

    def lean(w, k, q):
        w[k] = fix(0.6 * w[k] + 0.8 * w[q])

    w = {"embed": rnd(cfg["vocab"], W), "final.norm": one(W)}
    for i, ly in enumerate(cfg["layers"]):
        if ly.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", ly["mixer"]
        for q in (1, 2) if ly.get("mlp") else (1,):
            w[p + f"norm{q}"] = one(W)
            w[p + f"hc{q}.in"] = fix(1.0 / n + 0.3 * torch.randn(n, generator=gen))
            w[p + f"hc{q}.out"] = fix(1.0 + 0.3 * torch.randn(n, generator=gen))
            w[p + f"hc{q}.mix"] = fix(torch.eye(n) + 0.15 * torch.randn(n, n, generator=gen))
        if ly["type"] == "channel_delta":
            H, G, d, vd, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for t, c in (("q", G * d), ("k", G * d), ("v", H * vd)):
                w[p + f"mix.{t}"] = lin(c, W)
                w[p + f"mix.{t}.conv"] = rnd(c, taps, s=0.6)
            lean(w, p + "mix.k", p + "mix.q")
            lean(w, p + "mix.k.conv", p + "mix.q.conv")
            w[p + "mix.b"] = lin(H, W)
            w[p + "mix.A_log"] = rnd(H, s=0.7)
            w[p + "mix.dt_bias"] = fix(-2.0 + torch.randn(H * d, generator=gen))
            w[p + "mix.norm"] = one(vd)
            w[p + "mix.a1"], w[p + "mix.a2"] = lin(rank_a, W), lin(H * d, rank_a)
            w[p + "mix.g1"], w[p + "mix.g2"] = lin(rank_g, W), lin(H * vd, rank_g)
            w[p + "mix.o"] = lin(W, H * vd)
        else:
            l, r = m["left"], m["right"]
            H, G, d, vd, taps = l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["conv"]
            for t, c in (("q", H * d), ("k", G * d), ("v", G * vd)):
                w[p + f"mix.left.{t}"] = lin(c, W)
                w[p + f"mix.left.{t}.b"] = rnd(c, s=0.3)
                w[p + f"mix.left.{t}.conv"] = rnd(c, taps, s=0.6)
            w[p + "mix.left.q.norm"], w[p + "mix.left.k.norm"] = one(H * d), one(G * d)
            w[p + "mix.left.sink"] = fix(sink + torch.randn(H, generator=gen))
            w[p + "mix.left.o"], w[p + "mix.left.o.b"] = lin(W, H * vd), rnd(W, s=0.3)
            w[p + "mix.left.out"], w[p + "mix.right.out"] = one(W), one(W)
            H, d, vd = r["heads"], r["dim"], r["vdim"]
            for t, c in (("q", H * d), ("k", H * d), ("v", H * vd), ("g", H * vd), ("i", H), ("f", H)):
                w[p + f"mix.right.{t}"] = lin(c, W)
            lean(w, p + "mix.right.k", p + "mix.right.q")
            w[p + "mix.right.i.b"] = rnd(H, s=1.0)
            w[p + "mix.right.f.b"] = fix(3.0 + torch.randn(H, generator=gen))
            w[p + "mix.right.norm"] = one(H * vd)
            w[p + "mix.right.o"] = lin(W, H * vd)
        f = ly.get("mlp")
        if f and f["kind"] == "dense":
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = lin(f["ff"], W), lin(f["ff"], W), lin(W, f["ff"])
        elif f:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            w[p + "mlp.router"], w[p + "mlp.router.b"] = rnd(E, W, s=2.0 * W ** -0.5), rnd(E, s=0.3)
            for e in range(E):
                w[p + f"mlp.e{e}.gate"], w[p + f"mlp.e{e}.up"], w[p + f"mlp.e{e}.down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    return w

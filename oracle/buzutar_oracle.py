"""Plain fp32 restatement of the Buzutar design, one function per mechanism, slow on purpose.

Notation: W (width), V (vocab), T (new tokens of one sequence), pos0 (tokens before them).  Linear weights are
[out, in] and act as y = W x.  The residual stream starts as embed[token] * scale; a sublayer reads it as it is and
only its output is normed:

    x <- x + n1(mixer(x));   x <- x + n2(ff(x))          n(y) = y / sqrt(mean(y^2) + eps) * w

Mixers:

  attention            grouped-query attention without softmax and without positions.  One RMS norm spans all query
                       heads at once, another all key heads; the values are the keys as projected, before their norm.
                       Queries grow with their position by a logarithmic temperature.  A visible key weighs
                       sigmoid(scale q . k + b_h); weights are not normalised.  Output gate sigmoid(W_g x).
  latent_attention     queries and keys / values through RMS-normed low-rank latents.  A token leaves one row [c | r]
                       behind: c = the normed key / value latent, r = a rotated key part that all heads share.  Head h
                       scores (q_h^nope . U_k,h c_j + q_h^rot . r_j) * scale against the last `size` tokens and reads
                       U_v,h c_j through a softmax.  Interleaved rotary pairs with YaRN frequencies.  A layer may read
                       ANOTHER layer's rows (`kv_from`) with its own U_k, U_v.

Feed-forward: down relu(up x)^2.  Logits: a head of its own behind the final norm, capped by c tanh(z / c).

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


# ------------------------------------------------------------------------------------------ rotation

def yarn_ramp(dims: int, base: float, s: dict) -> torch.Tensor:
    """Per pair: 0 = the frequency stays, 1 = it is divided by the factor."""
    def pair_of(turns):          # the (fractional) pair that makes `turns` turns within the original length
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(s["fast"])), 0)
    hi = min(math.ceil(pair_of(s["slow"])), dims - 1)
    i = torch.arange(dims // 2, dtype=torch.float64)
    return ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)


def rotary_frequencies(rot: dict):
    """(frequency of every pair in double, factor on cos and sin)."""
    dims, base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = torch.tensor(base, dtype=torch.float64) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    if not s:
        return f, 1.0
    ramp = yarn_ramp(dims, base, s)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotary(x: torch.Tensor, pos: torch.Tensor, rot: dict) -> torch.Tensor:
    """x: [T, ..., d]; the pairs (2i, 2i + 1) of the first rot.dims numbers of the last axis are turned."""
    dims = rot["dims"]
    if dims == 0:
        return x
    f, m = rotary_frequencies(rot)
    a = pos.double().view(-1, 1) * f.view(1, -1)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    c, s = (a.cos() * m).float().view(shape), (a.sin() * m).float().view(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------ latent attention

def latent_rows(x: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float, pos0: int) -> torch.Tensor:
    """What T new tokens leave in a latent layer's cache: [T, kv_rank + rot_dim] = [normed latent | rotated shared key part]."""
    T, R, rd = x.shape[0], m["kv_rank"], m["rot_dim"]
    d = x @ p["dkv"].T
    c = rms_norm(d[:, :R], p["dkv.norm"], eps)
    return torch.cat([c, rotary(d[:, R:R + rd], torch.arange(pos0, pos0 + T), m["rot"])], -1)


def window_mask(pos: torch.Tensor, keys: int, size: Optional[int]) -> torch.Tensor:
    """[T, keys]: a position sees itself and the size - 1 tokens before it (size None: every earlier token)."""
    back = pos.view(-1, 1) - torch.arange(keys).view(1, -1)
    return (back >= 0) & (back < size) if size else back >= 0


def latent_attention(x: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float, pos0: int, rows: torch.Tensor) -> torch.Tensor:
    """The latent mixer over T new tokens; rows = cache rows [pos0 + T, kv_rank + rot_dim] of ALL tokens so far (this layer's own
    or, with kv_from, another layer's).  Keys and values are rebuilt per head, not absorbed."""
    T, H, d, rd, vd, R = x.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(pos0, pos0 + T)
    cq = rms_norm(x @ p["dq"].T, p["dq.norm"], eps)
    q = (cq @ p["uq"].T).view(T, H, d + rd)
    q_rot = rotary(q[..., d:], pos, m["rot"])
    c, r = rows[:, :R], rows[:, R:]
    k_nope = (c @ p["uk"].T).view(-1, H, d)
    v = (c @ p["uv"].T).view(-1, H, vd)
    vis = window_mask(pos, rows.shape[0], (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, vd)
    for h in range(H):
        s = (q[:, h, :d] @ k_nope[:, h].T + q_rot[:, h] @ r.T) * m["scale"]
        out[:, h] = torch.softmax(s.masked_fill(~vis, float("-inf")), -1) @ v[:, h]
    return out.reshape(T, H * vd) @ p["o"].T


# ------------------------------------------------------------------------------------------ sigmoid attention

def q_temperature(pos: torch.Tensor, t: Optional[dict]) -> torch.Tensor:
    if not t:
        return torch.ones(pos.shape[0])
    return (1.0 + t["coef"] * torch.log(torch.floor((pos.double() + 1.0) / t["every"]) + 1.0)).float()


def sigmoid_attention(x: torch.Tensor, p: Dict[str, torch.Tensor], m: dict, eps: float, pos0: int, keys: Optional[torch.Tensor]):
    """The sigmoid mixer over T new tokens; keys = projected (not normed) key rows of the tokens before them.  Returns (output, all
    key rows)."""
    T, H, G, d = x.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(pos0, pos0 + T)
    k_new = x @ p["k"].T
    k_all = k_new if keys is None else torch.cat([keys, k_new], 0)
    q = rms_norm(x @ p["q"].T, p["q.norm"], eps) * q_temperature(pos, m.get("q_temp")).view(-1, 1)
    k = rms_norm(k_all, p["k.norm"], eps).view(-1, G, d)
    v = k_all.view(-1, G, d)
    vis = window_mask(pos, k_all.shape[0], None)
    out = torch.zeros(T, H, d)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h * d:(h + 1) * d] @ k[:, g].T * m["scale"]
        out[:, h] = torch.where(vis, torch.sigmoid(s + p["pb"][h]), torch.zeros(())) @ v[:, g]
    return (out.reshape(T, H * d) * torch.sigmoid(x @ p["g"].T)) @ p["o"].T, k_all


def dense_ff(x, p):
    return torch.relu(x @ p["up"].T) ** 2 @ p["down"].T


def softcap(z: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return cap * torch.tanh(z / cap) if cap else z


def sub(params: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.float() for k, v in params.items() if k.startswith(prefix)}


class Buzutar:
    """The whole model over explicit per-request caches.  cfg: the dict of config.json; params: name -> tensor."""

    def __init__(self, cfg: dict, params: Dict[str, torch.Tensor]):
        self.cfg = cfg
        self.p = {k: v.float() for k, v in params.items()}
        self.eps = cfg["norm"]["eps"]

    def new_cache(self) -> dict:
        return {"len": 0, "rows": {}}

    def forward(self, tokens: List[int], cache: Optional[dict] = None, taps: Optional[list] = None) -> torch.Tensor:
        """Runs T new tokens of one request on top of `cache` (None: a whole prompt from an empty cache); returns logits [T, V]."""
        cfg, eps = self.cfg, self.eps
        if cache is None:
            cache = self.new_cache()
        pos0, rows = cache["len"], cache["rows"]
        x = self.p["embed"][torch.tensor(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
        for i, ly in enumerate(cfg["layers"]):
            lp = sub(self.p, f"l{i}.")
            mp, m = sub(lp, "mix."), ly["mixer"]
            if ly["type"] == "latent_attention":
                src = m.get("kv_from")
                if src is None:
                    new = latent_rows(x, mp, m, eps, pos0)
                    rows[i] = torch.cat([rows[i], new], 0) if i in rows else new
                    src = i
                y = latent_attention(x, mp, m, eps, pos0, rows[src])
            elif ly["type"] == "attention":
                y, rows[i] = sigmoid_attention(x, mp, m, eps, pos0, rows.get(i))
            else:
                raise ValueError(ly["type"])
            x = x + rms_norm(y, lp["norm1"], eps)
            if ly.get("mlp"):
                x = x + rms_norm(dense_ff(x, sub(lp, "mlp.")), lp["norm2"], eps)
            if taps is not None:
                taps.append(x.clone())
        cache["len"] = pos0 + len(tokens)
        return softcap(rms_norm(x, self.p["final.norm"], eps) @ self.p["head"].T, cfg.get("logit_softcap"))


# ------------------------------------------------------------------------------------------ small configurations

def latent_cfg(heads=4, dim=16, rot_dim=8, vdim=24, kv_rank=40, q_rank=48, scale=0.2, window=11, base=10000.0, scaling=None, kv_from=None) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(scaling)
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def attention_cfg(heads=4, kv_heads=2, dim=16, scale=0.25, coef=0.4, every=16) -> dict:
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "q_temp": {"coef": coef, "every": every}}}


def with_ff(layer: dict, ff: Optional[int] = 96) -> dict:
    layer = dict(layer)
    layer["mlp"] = {"kind": "dense", "ff": ff} if ff else None
    return layer


def make_config(vocab=200, width=96, layers=None, eps=1e-5, embed_scale=7.0, cap=20.0) -> dict:
    return {"architecture": "Buzutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "logit_softcap": cap, "layers": layers}


def make_weights(cfg: dict, seed: int = 0, bf16_values: bool = True, pb: float = -3.0) -> Dict[str, torch.Tensor]:
    """Random weights under the checkpoint's names; values bf16-representable by default so that the bf16 and fp32 paths load
    identical numbers.  pb: centre of the sigmoid heads' biases (weights are not normalised over keys)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def fix(t):
        return t.bfloat16().float() if bf16_values else t

    def rnd(*shape, s=1.0):
        return fix(torch.randn(*shape, generator=g) * s)

    def one(n):
        return fix(1.0 + 0.2 * torch.randn(n, generator=g))

    w = {"embed": rnd(cfg["vocab"], W, s=0.2), "head": rnd(cfg["vocab"], W, s=3.0 * W ** -0.5), "final.norm": one(W)}
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        w[p + "norm1"] = one(W)
        H, d = m["heads"], m["dim"]
        if ly["type"] == "latent_attention":
            rd, vd, R, Q = m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            w[p + "mix.dq"] = rnd(Q, W, s=W ** -0.5)
            w[p + "mix.dq.norm"] = one(Q)
            w[p + "mix.uq"] = rnd(H * (d + rd), Q, s=Q ** -0.5)
            if m.get("kv_from") is None:
                w[p + "mix.dkv"] = rnd(R + rd, W, s=W ** -0.5)
                w[p + "mix.dkv.norm"] = one(R)
            w[p + "mix.uk"] = rnd(H * d, R, s=R ** -0.5)
            w[p + "mix.uv"] = rnd(H * vd, R, s=R ** -0.5)
            w[p + "mix.o"] = rnd(W, H * vd, s=(H * vd) ** -0.5)
        else:
            G = m["kv_heads"]
            w[p + "mix.q"] = rnd(H * d, W, s=W ** -0.5)
            w[p + "mix.k"] = rnd(G * d, W, s=W ** -0.5)
            w[p + "mix.q.norm"] = one(H * d)
            w[p + "mix.k.norm"] = one(G * d)
            w[p + "mix.pb"] = fix(pb + torch.randn(H, generator=g))
            w[p + "mix.g"] = rnd(H * d, W, s=W ** -0.5)
            w[p + "mix.o"] = rnd(W, H * d, s=(H * d) ** -0.5)
        if ly.get("mlp"):
            w[p + "norm2"] = one(W)
            w[p + "mlp.up"] = rnd(ly["mlp"]["ff"], W, s=W ** -0.5)
            w[p + "mlp.down"] = rnd(W, ly["mlp"]["ff"], s=ly["mlp"]["ff"] ** -0.5)
    return w

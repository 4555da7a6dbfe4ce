"""Buzutar on the host: config.json through the registry's parser (every key, defaults, refusals), and the plain restatement against
itself - token by token, in portions - and against properties that hold by construction.  No GPU."""
import ctypes as C
import importlib
import json
import math

import pytest
import torch

from oracle import buzutar_oracle as Z


@pytest.fixture(scope="module")
def lib():
    return importlib.import_module("nano-vllm-candle_b200._lib").lib()


def parse(lib, cfg):
    h = C.c_void_p()
    rc = lib.nvc_model_config_from_json(json.dumps(cfg).encode(), C.byref(h))
    return rc, h, lib.nvc_model_config_last_error().decode()


SC = {"factor": 3.0, "original": 40, "fast": 5.0, "slow": 0.5}


def good():
    return Z.make_config(vocab=77, width=40, layers=[
        Z.with_ff(Z.latent_cfg(2, 8, 8, 12, 20, 24, window=7, scaling=SC), 64),
        Z.with_ff(Z.attention_cfg(6, 3, 8), None),
        Z.with_ff(Z.latent_cfg(3, 6, 8, 4, 20, 12, window=3, scaling=SC, kv_from=0), 24),
        Z.with_ff(Z.attention_cfg(2, 1, 12), 32),
    ])


def test_a_configuration_is_accepted_and_registered(lib):
    rc, h, err = parse(lib, good())
    assert rc == 0, err
    assert lib.nvc_model_config_architecture(h).decode() == "Buzutar"
    assert lib.nvc_model_config_vocab(h) == 77
    layers = (C.c_int32 * 8)()
    assert lib.nvc_model_config_layer_runs(h, layers, None, None, 8) == 4 and list(layers)[:4] == [0, 1, 2, 3]
    lib.nvc_model_config_free(h)


@pytest.mark.parametrize("mutate,needle", [
    (lambda c: c["layers"][0].update(type="delta"), "not supported"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(scaling=[1]), "rot.scaling"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "positive"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "cache of its own"),            # not a latent layer
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(scaling=None), "must equal"),        # another rotation
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=24), "must equal"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=9), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda c: c["layers"][3]["mlp"].update(kind="moe"), "dense"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c.update(embedding=3), "embedding"),
    (lambda c: c.pop("norm"), "norm.eps"),
])
def test_what_the_parser_refuses(lib, mutate, needle):
    c = good()
    mutate(c)
    rc, _, err = parse(lib, c)
    assert rc != 0 and needle in err, err


def test_absent_keys_mean_absent_mechanisms(lib):
    c = good()
    c["layers"][0]["mixer"].pop("mask")
    c["layers"][2]["mixer"]["mask"] = None
    c["layers"][1]["mixer"].pop("q_temp")
    c["layers"][0]["mixer"]["rot"].pop("scaling")
    c["layers"][2]["mixer"]["rot"]["scaling"] = None
    c["logit_softcap"] = None
    c.pop("embedding")
    c["layers"][3]["mlp"] = None
    rc, h, err = parse(lib, c)
    assert rc == 0, err
    lib.nvc_model_config_free(h)


def test_families_without_scaled_frequencies_refuse_them(lib):
    from oracle import fefozen_oracle as F
    c = F.make_config(vocab=50, width=32, layers=[F.with_dense(F.latent_cfg(), 32)])
    c["layers"][0]["mixer"]["rot"]["scaling"] = SC
    rc, _, err = parse(lib, c)
    assert rc != 0 and "scaling" in err


# ------------------------------------------------------------------------------------------ the plain restatement
def test_portions_and_single_tokens_give_the_whole_prompts_logits():
    cfg = good()
    m = Z.Buzutar(cfg, Z.make_weights(cfg, 1))
    p = torch.randint(0, 77, (40,), generator=torch.Generator().manual_seed(2)).tolist()
    whole = m.forward(p)
    for cuts in ([1] * 40, [2, 7, 1, 13, 17], [39, 1]):
        cache, got, at = m.new_cache(), [], 0
        for n in cuts:
            got.append(m.forward(p[at:at + n], cache))
            at += n
        assert torch.allclose(torch.cat(got), whole, atol=2e-4)
    assert whole.abs().max() <= cfg["logit_softcap"]


def test_the_windows_mask():
    v = Z.window_mask(torch.tensor([0, 4, 9]), 10, 3)
    assert v[0].nonzero().flatten().tolist() == [0]
    assert v[1].nonzero().flatten().tolist() == [2, 3, 4] and v[2].nonzero().flatten().tolist() == [7, 8, 9]
    assert Z.window_mask(torch.tensor([4]), 10, None)[0].sum() == 5


def test_scaled_frequencies_between_the_bounds():
    rot = {"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}}
    f, m = Z.rotary_frequencies(rot)
    plain = torch.tensor(10000.0, dtype=torch.float64) ** (-2.0 * torch.arange(16, dtype=torch.float64) / 32)
    assert torch.allclose(f[:1], plain[:1]) and torch.allclose(f[-1:], plain[-1:] / 8.0)       # fast pairs stay, slow ones are stretched
    assert ((f <= plain) & (f >= plain / 8.0)).all() and (f[1:] < f[:-1]).all()
    assert m == 0.1 * math.log(8.0) + 1.0


def test_a_negligible_bias_silences_a_head():
    cfg = Z.make_config(vocab=30, width=24, layers=[Z.with_ff(Z.attention_cfg(2, 1, 8), None)])
    w = Z.make_weights(cfg, 3)
    x = torch.randn(6, 24, generator=torch.Generator().manual_seed(1))
    p, m = Z.sub(w, "l0.mix."), cfg["layers"][0]["mixer"]
    p["pb"] = torch.tensor([-1e4, -1e4])
    y, _ = Z.sigmoid_attention(x, p, m, 1e-5, 0, None)
    assert (y == 0).all()
    p["pb"] = torch.tensor([1e4, 1e4])                       # every visible key counts fully: the running sum of the keys
    p["g"] = torch.zeros_like(p["g"])
    p["o"] = torch.eye(24)[:, :16].contiguous()
    y, keys = Z.sigmoid_attention(x, p, m, 1e-5, 0, None)
    assert torch.allclose(y[:, :8], 0.5 * keys.cumsum(0), atol=1e-5) and torch.allclose(y[:, 8:16], 0.5 * keys.cumsum(0), atol=1e-5)

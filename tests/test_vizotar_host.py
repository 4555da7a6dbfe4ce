"""Vizotar on the host: config.json through the registry's parser (every key, defaults, refusals, layers that run another layer's
weights) and the plain restatement against itself (a whole prompt equals portions and token-by-token decoding).  No GPU."""
import ctypes as C
import importlib
import json

import pytest
import torch

from oracle import vizotar_oracle as Z

YARN = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}


@pytest.fixture(scope="module")
def lib():
    return importlib.import_module("nano-vllm-candle_b200._lib").lib()


def parse(lib, cfg):
    h = C.c_void_p()
    rc = lib.nvc_model_config_from_json(json.dumps(cfg).encode(), C.byref(h))
    return rc, h, lib.nvc_model_config_last_error().decode()


def good():
    layers = [
        Z.with_moe(Z.parallel_cfg(scaling=YARN), 5, 2, 24),
        Z.with_dense(Z.delta_cfg(), 40, 0.7),
        Z.with_none(Z.parallel_cfg(heads=2, kv_heads=2, dim=8, vdim=12, conv=1, window=5, rot_dims=8, mheads=1, mdim=4, mvdim=40)),
    ]
    layers += [Z.again(layers, 1), Z.again(layers, 0), Z.again(layers, 1)]
    return Z.make_config(vocab=77, width=40, streams=3, layers=layers)


def runs(lib, h, n=16):
    layers, passes, readd = (C.c_int32 * n)(), (C.c_int32 * n)(), (C.c_int32 * n)()
    k = lib.nvc_model_config_layer_runs(h, layers, passes, readd, n)
    assert not any(list(readd)[:k])
    return list(zip(list(layers)[:k], list(passes)[:k]))


def test_a_configuration_is_accepted_and_registered(lib):
    rc, h, err = parse(lib, good())
    assert rc == 0, err
    assert lib.nvc_model_config_architecture(h).decode() == "Vizotar"
    assert lib.nvc_model_config_vocab(h) == 77
    assert runs(lib, h) == [(0, 0), (1, 0), (2, 0), (1, 1), (0, 1), (1, 2)]
    lib.nvc_model_config_free(h)


def test_weights_of_may_name_a_later_layer_or_one_that_borrows_itself(lib):
    c = good()
    c["layers"][0] = {**c["layers"][1], "weights_of": 3}       # 3 borrows from 1
    c["layers"][4] = {**c["layers"][2], "weights_of": 2}
    rc, h, err = parse(lib, c)
    assert rc == 0, err
    assert runs(lib, h) == [(1, 0), (1, 1), (2, 0), (1, 2), (2, 1), (1, 3)]
    lib.nvc_model_config_free(h)


def broken(mutate):
    c = good()
    mutate(c)
    return c


@pytest.mark.parametrize("mutate,needle", [
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.update(streams=17), "streams"),
    (lambda c: c.pop("norm"), "norm.eps"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="attention"), "not supported"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(conv=40), "taps"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=64), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=-1.0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "not supported"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(experts=300), "256"),
    (lambda c: c["layers"][3].update(weights_of=3), "another layer"),
    (lambda c: c["layers"][3].update(weights_of=9), "another layer"),
    (lambda c: (c["layers"][3].update(weights_of=4), c["layers"][4].update(weights_of=3)), "circle"),
])
def test_what_the_parser_refuses(lib, mutate, needle):
    rc, h, err = parse(lib, broken(mutate))
    assert rc != 0 and needle in err, err


def test_absent_keys_mean_absent_mechanisms(lib):
    c = good()
    left = c["layers"][0]["mixer"]["left"]
    left.pop("mask")                                      # every earlier token is visible
    left["rot"]["scaling"] = None                         # plain frequencies
    c["layers"][2]["mixer"]["left"]["rot"] = None         # no positions
    c["layers"][1]["weights_of"] = None                   # tensors of its own
    rc, h, err = parse(lib, c)
    assert rc == 0, err
    lib.nvc_model_config_free(h)


@pytest.mark.parametrize("streams", [1, 3])
def test_the_restatement_agrees_with_itself_however_the_prompt_is_cut(streams):
    cfg = {**good(), "streams": streams}
    m = Z.Vizotar(cfg, Z.make_weights(cfg, 3))
    p = torch.randint(0, 77, (40,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = m.forward(p)
    for sizes in ([1] * 40, [2, 3, 1, 11, 5, 18], [39, 1]):
        cache, rows, at = m.new_cache(), [], 0
        for n in sizes:
            rows.append(m.forward(p[at:at + n], cache))
            at += n
        assert (torch.cat(rows) - whole).abs().max() < 1e-3


def test_one_stream_with_unit_weights_is_the_plain_residual_sum():
    """Hyper-connections with one stream, in = mix = out = 1 are x + f(norm(x)): the restatement with them equals a loop without."""
    cfg = Z.make_config(vocab=50, width=32, streams=1, layers=[Z.with_dense(Z.delta_cfg())])
    w = Z.make_weights(cfg, 1)
    for q in (1, 2):
        for n in ("in", "out", "mix"):
            w[f"l0.hc{q}.{n}"] = torch.ones_like(w[f"l0.hc{q}.{n}"])
    p = list(range(12))
    x = w["embed"][torch.tensor(p)]
    y, _ = Z.channel_delta_mixer(Z.rms_norm(x, w["l0.norm1"], 1e-5), Z.sub(w, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5, None)
    x = x + y
    x = x + Z.dense_ff(Z.rms_norm(x, w["l0.norm2"], 1e-5), Z.sub(w, "l0.mlp."), cfg["layers"][0]["mlp"]["limit"])
    assert torch.allclose(Z.Vizotar(cfg, w).forward(p), Z.rms_norm(x, w["final.norm"], 1e-5) @ w["embed"].T, rtol=1e-4, atol=1e-4)

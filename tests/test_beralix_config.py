"""The Beralix configuration (keys, defaults, errors, what it asks of weights and cache) and the plain
implementation's mechanisms against other ways of computing them, on the CPU."""
import copy
import math

import numpy as np
import pytest
import torch

from beralix_tiny import CONFIGS, make_weights, ramp, random_config, rotation, tensor_shapes, tokens_of, write_folder
from plain import beralix_plain as plain
from torchless_rs_b200.cache.requests import PagedKVRequest, PagedLatentRequest, StateRequest
from torchless_rs_b200.config import BeralixConfig, ConfigError, config_from_dict, load_config
from torchless_rs_b200.engine.model import expected_tensors
from torchless_rs_b200.parts import lookup
from torchless_rs_b200.parts.position import RotaryHalfSplit


@pytest.mark.parametrize("name", ["P", "Q", "R", 1, 2, 3, 4, 5])
def test_reads_back_and_asks_for_the_design_s_tensors(name):
    d = CONFIGS[name] if isinstance(name, str) else random_config(name)
    cfg = config_from_dict(d)
    assert isinstance(cfg, BeralixConfig)
    assert config_from_dict(cfg.to_dict()) == cfg
    want = expected_tensors(cfg.model_spec())
    shapes = tensor_shapes(d)
    assert {k: tuple(v.shape) for k, v in want.items() if k in shapes} == shapes
    assert all(v.optional for k, v in want.items() if k not in shapes)
    assert cfg.model_spec().logit_softcap == d.get("logit_softcap")


def test_loads_a_folder(tmp_path):
    cfg = CONFIGS["P"]
    d = write_folder(cfg, make_weights(cfg, 0, torch.bfloat16), str(tmp_path))
    assert load_config(d).width == 96
    from torchless_rs_b200.weights.loader import load_checked
    w, _ = load_checked(d, expected_tensors(load_config(d).model_spec()))
    assert w["l0.mix.vmix"].shape == ()


def test_the_first_layer_that_mixes_gives_its_values():
    spec = config_from_dict(CONFIGS["Q"]).model_spec()
    assert [l.mixer.get("value_mix") for l in spec.layers] == [None, None, None, "first", None, "later", None]
    want = expected_tensors(spec)
    assert want["l3.mix.vmix"].optional and not want["l5.mix.vmix"].optional
    assert "l1.mix.vmix" not in want


def test_what_the_mixers_ask_of_the_cache():
    class Rt:      # a mixer is built without a device up to its weights
        is_f32, act_dtype, device = True, torch.float32, torch.device("cpu")
    reqs = []
    for l in config_from_dict(CONFIGS["P"]).model_spec().layers:
        pos = lookup("position", l.position.kind)(l.position, Rt) if l.position else None
        reqs.append(lookup("mixer", l.mixer.kind)(l.mixer, "x", Rt, position=pos).cache_request())
    assert reqs[0] == PagedKVRequest(2, 20, 20, v_head_dim=12)
    assert reqs[1] == (StateRequest((40, 6), torch.float32), StateRequest((3, 40), torch.float32))
    assert reqs[2] == PagedLatentRequest(24 + 8, None)
    assert reqs[3] == PagedKVRequest(2, 16, 70, v_head_dim=12)


def _broken(change):
    d = copy.deepcopy(CONFIGS["P"])
    change(d)
    return d


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0].update(type="nothing"), "nothing"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=22), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda d: d["layers"][2]["mixer"]["rot"].update(dims=4), "dims"),
    (lambda d: d["layers"][1]["mixer"].pop("dt_rank"), "dt_rank"),
    (lambda d: d["layers"][3]["mixer"].update(vdim=10), "mixed"),
    (lambda d: d["layers"][0]["mlp"].update(kind="sparse"), "sparse"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d.update(layers=[]), "layers"),
])
def test_errors_name_the_key(change, word):
    with pytest.raises(ConfigError, match=word):
        config_from_dict(_broken(change))


@pytest.mark.parametrize("rot", [
    rotation(16, 10000.0), rotation(32, 500000.0, ramp(8.0, 4096)), rotation(6, 100.0, ramp(2.0, 32, 4.0, 1.0)),
    rotation(8, 10000.0, ramp(4.0, 7, 32.0, 1.0)),        # original so short that both ends lie before the first pair
    rotation(4, 10.0, ramp(16.0, 1 << 20, 2.0, 1.0)),     # so long that both lie behind the last
    rotation(2, 10000.0, ramp(1.0, 64))])
def test_frequencies_and_amplitude(rot):
    f, amp = plain.frequencies(rot, rot["dims"])
    params = {"head_dim": rot["dims"], "theta": rot["base"]}
    if rot.get("scaling"):
        params["scaling"] = {"kind": "ramp", **rot["scaling"]}

    class Rt:
        device = torch.device("cpu")
    from torchless_rs_b200.config import PartSpec
    part = RotaryHalfSplit(PartSpec("rope_half_split", params), Rt)
    assert np.allclose(part.inv_freq.numpy(), f, rtol=1e-6) and abs(part.amplitude - amp) < 1e-12
    if rot.get("scaling"):
        plainly = np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])
        factor = rot["scaling"]["factor"]
        assert (f <= plainly * (1 + 1e-12)).all() and (f >= plainly / factor * (1 - 1e-12)).all()
        assert abs(amp - (0.1 * math.log(factor) + 1)) < 1e-12


# ---- the plain implementation against other computations ---------------------------------------------------

def test_plain_layer_norm():
    rng = np.random.default_rng(0)
    x, w, b = rng.normal(3, 2, (5, 33)), rng.normal(size=33), rng.normal(size=33)
    ref = torch.nn.functional.layer_norm(torch.tensor(x), (33,), torch.tensor(w), torch.tensor(b), 1e-4).numpy()
    assert np.allclose(plain.layer_norm(x, w, b, 1e-4), ref, atol=1e-12)


def test_plain_rotation_depends_on_distance_only_and_carries_the_factor():
    rng = np.random.default_rng(1)
    f, amp = plain.frequencies(rotation(8, 1000.0, ramp(4.0, 64, 8.0, 1.0)), 8)
    q, k = rng.normal(size=(1, 12)), rng.normal(size=(1, 12))
    turn = lambda x, p: plain.rotate_halves(x, np.array([float(p)]), f, amp)[0]
    assert abs(turn(q, 70) @ turn(k, 61) - turn(q, 9) @ turn(k, 0)) < 1e-9
    assert abs(np.linalg.norm(turn(q, 5)[:8]) - amp * np.linalg.norm(q[0, :8])) < 1e-9
    assert (turn(q, 5)[8:] == q[0, 8:]).all()


def test_plain_selective_scan_in_closed_form():
    """y_t = sum over s <= t of exp(A (dt_(s+1) + ... + dt_t)) dt_s x_s (B_s . C_t entry by entry) + D x_t."""
    rng = np.random.default_rng(2)
    n, C, N = 13, 5, 4
    x, dt = rng.normal(size=(n, C)), rng.uniform(0.01, 1, (n, C))
    A, B, Cm, D = -rng.uniform(0.1, 3, (C, N)), rng.normal(size=(n, N)), rng.normal(size=(n, N)), rng.normal(size=C)
    y, S = plain.selective_scan(x, dt, A, B, Cm, D)
    cum = np.cumsum(dt, axis=0)
    for t in range(n):
        want = D * x[t]
        for s in range(t + 1):
            want = want + (np.exp((cum[t] - cum[s])[:, None] * A) * B[s] * Cm[t]).sum(1) * dt[s] * x[s]
        assert np.allclose(y[t], want, atol=1e-10)
    y2, S2 = plain.selective_scan(x[6:], dt[6:], A, B[6:], Cm[6:], D, plain.selective_scan(x[:6], dt[:6], A, B[:6], Cm[:6], D)[1])
    assert np.allclose(y2, y[6:]) and np.allclose(S2, S)


def test_plain_convolution():
    rng = np.random.default_rng(3)
    x, w, b = rng.normal(size=(9, 4)), rng.normal(size=(4, 3)), rng.normal(size=4)
    pad = torch.nn.functional.pad(torch.tensor(x.T[None]), (2, 0))
    ref = torch.nn.functional.conv1d(pad, torch.tensor(w[:, None]), torch.tensor(b), groups=4)[0].numpy().T
    assert np.allclose(plain.short_convolution(x, w, b), ref, atol=1e-12)


def test_plain_window_and_cap():
    m = plain.visible(6, 3)
    assert m[4].tolist() == [False, False, True, True, True, False]
    assert plain.visible(4, None).sum() == 10 and plain.visible(4, 1).sum() == 4
    z = np.array([-1000.0, 0.0, 0.1, 1000.0])
    assert np.allclose(plain.soft_cap(z, 5.0), [-5, 0, 5 * math.tanh(0.02), 5]) and (plain.soft_cap(z, None) == z).all()


@pytest.mark.parametrize("name", ["P", "Q", "R"])
def test_plain_model_is_causal_and_every_mechanism_counts(name):
    cfg = CONFIGS[name]
    w = {k: v.double().numpy() for k, v in make_weights(cfg, 1, torch.float32).items()}
    toks = tokens_of(np.random.default_rng(4), 40, cfg["vocab"])
    ref = plain.forward(cfg, w, toks)
    assert np.allclose(plain.forward(cfg, w, toks[:25]), ref[:25], atol=1e-10)
    for key in w:
        first_mix = next((i for i, l in enumerate(cfg["layers"]) if l["mixer"].get("v_mix")), None)
        layer = cfg["layers"][int(key[1:key.index(".")])] if key[0] == "l" else {"mixer": {}}
        if key == f"l{first_mix}.mix.vmix" or \
                (layer["mixer"].get("mask") == {"size": 1} and key.endswith((".mix.q", ".mix.k"))):
            continue                                    # stored, but not used; a softmax over one key
        changed = dict(w)
        changed[key] = w[key] + 0.1 * (1.0 + np.abs(w[key])) * np.random.default_rng(5).choice([-1.0, 1.0], np.shape(w[key]))
        assert np.abs(plain.forward(cfg, changed, toks) - ref).max() > 1e-4, f"{key} does not reach the logits"

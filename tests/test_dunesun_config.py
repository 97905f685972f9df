"""The Dunesun configuration, its tensor list, the order of its layers with what is added before a pass, what
its parts ask of the cache, and the plain implementation's mechanisms against closed forms (no device needed)."""
import copy

import numpy as np
import pytest
import torch

import torchless_rs_b200 as tl
from dunesun_tiny import CONFIGS, random_config, tensor_shapes
from plain import dunesun_plain as plain
from torchless_rs_b200.cache import Cache, PAGE, PagedKVRequest, StateRequest
from torchless_rs_b200.config import ConfigError, PassStart
from torchless_rs_b200.engine.model import expected_tensors

ALL = {**CONFIGS, **{f"seed{s}": random_config(s) for s in range(1, 9)}}


@pytest.mark.parametrize("name", sorted(ALL))
def test_keys_are_read_and_written_back(name):
    raw = ALL[name]
    cfg = tl.config_from_dict(raw)
    assert type(cfg).__name__ == "DunesunConfig"
    assert tl.config_from_dict(cfg.to_dict()) == cfg
    assert (cfg.width, cfg.vocab, cfg.eps, cfg.logit_scale, cfg.max_positions) == \
        (raw["width"], raw["vocab"], raw["norm"]["eps"], raw["logit_scale"], raw["max_positions"])
    if raw.get("loop"):
        assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == tuple(raw["loop"][k] for k in ("start", "stop", "times"))
    else:
        assert cfg.loop is None
    for layer, entry in zip(cfg.layers, raw["layers"]):
        m, got = entry["mixer"], layer.mixer
        assert got.type == entry["type"]
        if got.type == "attention":
            assert (got.heads, got.kv_heads, got.dim, got.vdim, got.scale) == \
                tuple(m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
            assert got.window == (m.get("mask") or {}).get("size")
        else:
            assert got.to_dict() == m
        if entry["mlp"] is None:
            assert layer.mlp is None
        else:
            assert layer.mlp.to_dict() == entry["mlp"]


def test_errors_name_the_key():
    base = CONFIGS["A"]
    L = lambda c, i: c["layers"][i]
    for change, word in ((lambda c: L(c, 0).__setitem__("type", "mamba3"), "type"),
                         (lambda c: L(c, 0)["mlp"].__setitem__("kind", "dense"), "kind"),
                         (lambda c: L(c, 0)["mlp"].pop("router"), "router"),
                         (lambda c: L(c, 0)["mlp"]["expert"].pop("ff"), "ff"),
                         (lambda c: L(c, 0)["mlp"]["router"].__setitem__("top", 7), "top"),
                         (lambda c: L(c, 0)["mixer"].pop("state"), "state"),
                         (lambda c: L(c, 0)["mixer"].__setitem__("groups", 2), "groups"),
                         (lambda c: L(c, 0)["mixer"].__setitem__("norm_groups", 5), "norm_groups"),
                         (lambda c: L(c, 0)["mixer"].__setitem__("conv", 0), "conv"),
                         (lambda c: L(c, 1)["mixer"].pop("scale"), "scale"),
                         (lambda c: L(c, 1)["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
                         (lambda c: L(c, 1)["mixer"]["mask"].__setitem__("size", 0), "size"),
                         (lambda c: c["loop"].__setitem__("stop", 5), "stop"),
                         (lambda c: c["loop"].__setitem__("start", 3), "start"),
                         (lambda c: c["loop"].__setitem__("times", 0), "times"),
                         (lambda c: c["norm"].pop("eps"), "eps"),
                         (lambda c: c.pop("max_positions"), "max_positions"),
                         (lambda c: c.pop("width"), "width")):
        c = copy.deepcopy(base)
        change(c)
        with pytest.raises(ConfigError) as e:
            tl.config_from_dict(c)
        assert word in str(e.value)


@pytest.mark.parametrize("name", sorted(ALL))
def test_the_model_asks_for_the_designs_tensors(name):
    exp = expected_tensors(tl.config_from_dict(ALL[name]).model_spec())
    assert {n: tuple(s.shape) for n, s in exp.items()} == tensor_shapes(ALL[name])
    assert not any(s.optional for s in exp.values())


def test_order_and_what_is_added_before_a_pass():
    spec = tl.config_from_dict(CONFIGS["A"]).model_spec()          # layers 1 and 2 three times
    assert spec.order == (0, 1, 2, 1, 2, 1, 2, 3)
    assert spec.pass_starts == {1: PassStart(0, False), 3: PassStart(1, True), 5: PassStart(2, True)}
    assert (spec.pass_table_name, spec.pass_rows) == ("loop.step", 3)
    spec = tl.config_from_dict(CONFIGS["B"]).model_spec()          # no run is repeated
    assert spec.order == (0, 1, 2, 3) and not spec.pass_starts and spec.pass_table_name is None
    spec = tl.config_from_dict(CONFIGS["C"]).model_spec()          # all layers twice
    assert spec.order == (0, 1, 2, 3, 0, 1, 2, 3)
    assert spec.pass_starts == {0: PassStart(0, False), 4: PassStart(1, True)}
    for name, raw in ALL.items():
        spec = tl.config_from_dict(raw).model_spec()
        want = plain.run_order(len(raw["layers"]), raw.get("loop"))
        assert [i for i, _ in want] == list(spec.order), name
        assert {k: t for k, (_, t) in enumerate(want) if t is not None} == {k: s.row for k, s in spec.pass_starts.items()}


def test_a_pass_start_that_fits_nothing_is_an_error():
    import dataclasses
    spec = tl.config_from_dict(CONFIGS["A"]).model_spec()
    for starts in ({8: PassStart(0)}, {1: PassStart(3)}):
        with pytest.raises(ConfigError):
            dataclasses.replace(spec, pass_starts=starts).validate()
    with pytest.raises(ConfigError):
        dataclasses.replace(spec, streams=2).validate()


def test_parts_and_what_they_ask_of_the_cache():
    from torchless_rs_b200.parts import lookup
    spec = tl.config_from_dict(CONFIGS["A"]).model_spec()
    assert not spec.tie_head_to_embedding and spec.position_table_name == "pos" and spec.max_positions == 1024
    assert spec.final_norm.kind == "rmsnorm_one_plus" and spec.final_norm.params["output_scale"] == 0.7
    kinds = [(l.block.kind, l.mixer.kind, l.feed_forward.kind) for l in spec.layers]
    assert kinds == [("parallel_sublayers", "mamba2", "moe_softmax_chosen"),
                     ("parallel_sublayers", "sink_window_attention", "moe_softmax_chosen"),
                     ("parallel_sublayers", "mamba2", "none"),
                     ("parallel_sublayers", "sink_window_attention", "moe_softmax_chosen")]
    a = spec.layers[1].mixer.params
    assert a["sink"] == 0.0 and a["qk_norm"] == "whole" and not a["bias"] and not a["gate"] and a["window"] == 20
    f = spec.layers[0].feed_forward.params
    assert (f["experts"], f["top"], f["ff"], f["shared_ff"]) == (6, 2, 40, 56)
    assert all(lookup("mixer", l.mixer.kind).graph_safe for l in spec.layers)
    # every pass keeps its own pages and states
    kv = PagedKVRequest(2, 16, 20, v_head_dim=16)
    ssm = (StateRequest((4, 16, 16)), StateRequest((1, 4 * 16 + 2 * 2 * 16)))
    c = Cache([kv, ssm, kv, ssm], max_tokens=4 * PAGE, max_slots=3, dtype=torch.float32, device="cpu")
    assert c.view(0).k_pages.data_ptr() != c.view(2).k_pages.data_ptr() and c.view(0).group is c.view(2).group
    for j in (0, 1):
        assert c.view(1)[j].data_ptr() != c.view(3)[j].data_ptr()
        c.view(1)[j].fill_(2.0)
        c.view(3)[j].fill_(3.0)
    s = c.acquire(1)[0]
    assert all(float(c.view(k)[j][s].abs().sum()) == 0.0 for k in (1, 3) for j in (0, 1))


def test_a_mixer_holds_rows_for_the_feed_forward_beside_it():
    from torchless_rs_b200.parts.linear import InputRows

    class Rt:
        stack = staticmethod(lambda mats: torch.cat(list(mats)))
    m = InputRows()
    w = {"router": torch.full((3, 4), 2.0), "gate": torch.full((1, 4), 3.0)}
    m.take_rows(["router", "gate"])
    got = m.stack_input(Rt, w, [torch.ones(5, 4), torch.ones(2, 4)])
    assert (m.own_rows, m.taken_rows) == (7, 4) and got.shape == (16, 4)
    assert got[:, 0].tolist() == [1.0] * 7 + [2.0] * 3 + [3.0] + [0.0] * 5


# ---- the plain mechanisms against closed forms --------------------------------------------------------------
def test_plain_window_and_softmax_with_one_added():
    vis = plain.visible(9, 3)
    for i in range(9):
        assert [j for j in range(9) if vis[i, j]] == list(range(max(0, i - 2), i + 1))
    assert plain.visible(4, None).sum() == 10
    p = plain.softmax_plus_one(np.array([[0.0, 0.0, 5.0]]), np.array([[True, True, False]]))
    assert np.allclose(p, [[1 / 3, 1 / 3, 0.0]])
    p = plain.softmax_plus_one(np.array([[-800.0, -801.0]]), np.array([[True, True]]))
    assert np.allclose(p, 0.0)                      # the added one takes all
    p = plain.softmax_plus_one(np.array([[800.0, 799.0]]), np.array([[True, True]]))
    assert np.allclose(p, [[1 / (1 + np.exp(-1)), 1 / (1 + np.exp(1))]])


def test_plain_convolution_and_recurrence():
    rng = np.random.default_rng(0)
    x, w, b = rng.normal(size=(6, 2)), rng.normal(size=(2, 3)), rng.normal(size=2)
    y = plain.short_convolution(x, w, b)
    assert np.allclose(y[0], b + w[:, 2] * x[0])
    assert np.allclose(y[4], b + w[:, 0] * x[2] + w[:, 1] * x[3] + w[:, 2] * x[4])
    # the recurrence as its unrolled sum
    n, H, G, N, P = 7, 4, 2, 3, 5
    xs, B, C = rng.normal(size=(n, H, P)), rng.normal(size=(n, G, N)), rng.normal(size=(n, G, N))
    dt, A, D = rng.uniform(0.1, 1.0, (n, H)), rng.normal(size=H), rng.normal(size=H)
    y = plain.selective_scan(xs, B, C, dt, A, D)
    for h in range(H):
        g = h // 2
        for t in range(n):
            want = D[h] * xs[t, h]
            for s in range(t + 1):
                decay = np.exp(-np.exp(A[h]) * dt[s + 1:t + 1, h].sum())
                want = want + decay * dt[s, h] * (B[s, g] @ C[t, g]) * xs[s, h]
            assert np.allclose(y[t, h], want)


def test_plain_gate_norm_router_and_passes():
    rng = np.random.default_rng(1)
    y, z, w = rng.normal(size=(3, 6)), rng.normal(size=(3, 6)), rng.normal(size=6)
    got = plain.gated_group_norm(y, z, w, 2, 1e-3)
    g = y * z / (1 + np.exp(-z))
    for part in (slice(0, 3), slice(3, 6)):
        assert np.allclose(got[:, part], g[:, part] / np.sqrt((g[:, part] ** 2).mean(-1, keepdims=True) + 1e-3) * w[part])
    idx, wt = plain.route(np.array([[1.0, 3.0, 3.0, -2.0]]), 2)
    assert idx.tolist() == [[1, 2]] and np.allclose(wt, 0.5)
    idx, wt = plain.route(np.array([[0.0, np.log(3.0), -9.0]]), 2)
    assert idx.tolist() == [[1, 0]] and np.allclose(wt, [[0.75, 0.25]])
    e, tab = np.ones((2, 3)), np.arange(6.0).reshape(2, 3)
    assert np.allclose(plain.pass_start(5 * e, e, tab, 0), 5 + tab[0]) and np.allclose(plain.pass_start(5 * e, e, tab, 1), 6 + tab[1])

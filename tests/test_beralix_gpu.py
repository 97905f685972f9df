"""The Beralix decoder in the engine against the plain implementation: whole prompts, prefill against
token-by-token decoding, portions down to two tokens, unequal batches, slots, pages and state used
again, long decoding, greedy generation through the entry point, the replay program and the command
line; then each mechanism's kernels alone on inputs made so that a wrong window edge, a missed far
key, a lost state or a convolution that looks past a sequence's start shows."""
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from beralix_tiny import CONFIGS, BModel, make_weights, ramp, random_config, rotation, tokens_of, write_folder
from plain import beralix_plain as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = [(c, d) for c in ("P", "Q", "R") for d in ("float32", "bfloat16")]


def assert_close(got, ref, dtype, what=""):
    """32-bit: rounding through the layers is a few 1e-6 of the largest logit (capped or around 10); the bound per
    logit is 2e-5 of the largest + 1e-4 |ref|.  bfloat16: an activation is rounded to 8 bits at a dozen places per
    layer, and a row whose softmax is sharp turns that into a few percent of its logits; the bound is 2 % of the
    logits' root mean square over all rows and 10 % of the largest logit for any one.  What a mechanism's fault
    does shows in the 32-bit run and in the kernels alone."""
    assert got.shape == ref.shape and np.isfinite(got).all(), what
    err = got - ref
    if dtype == "float32":
        bad = np.abs(err) > 2e-5 * max(1.0, np.abs(ref).max()) + 1e-4 * np.abs(ref)
        assert not bad.any(), (f"{what}: max err {np.abs(err).max():.3e} of {np.abs(ref).max():.1f} "
                               f"(first bad row {np.argwhere(bad)[0]})")
        return
    rms = float(np.sqrt((err ** 2).mean()) / np.sqrt((ref ** 2).mean()))
    worst = float(np.abs(err).max() / np.abs(ref).max())
    assert rms <= 2e-2 and worst <= 1e-1, f"{what}: rms error {rms:.3e} of the logits' rms, worst logit {worst:.3e}"


def _feed(tm, slot, toks, cuts):
    """Feeds `toks` to one sequence in pieces of the sizes `cuts` (the rest one by one) and returns the
    logits of every position."""
    rows, at = [], 0
    for c in list(cuts) + [1] * len(toks):
        if at >= len(toks):
            break
        piece = toks[at:at + c]
        rows.append(tm.step_np([slot], [piece], "all"))
        at += len(piece)
    return np.concatenate(rows)


@pytest.mark.parametrize("name,dtype", BOTH)
def test_whole_prompt_and_decoding_and_portions(name, dtype):
    tm = BModel(name, dtype, seed=3)
    rng = np.random.default_rng(11)
    toks = tokens_of(rng, 150, tm.cfg["vocab"])
    ref = tm.reference(toks)
    for cuts, what in (([150], "whole"), ([40], "prefix, then one by one across windows and page borders"),
                       ([2, 3, 59, 2, 64, 1, 17, 2], "portions"), ([], "from the first token one by one"),
                       ([63, 2, 63, 2], "portions that end at and start on page borders"),
                       ([1, 1, 1, 2, 2], "portions shorter than the convolutions")):
        s = tm.engine.start_sequences(1)
        got = _feed(tm, s[0], toks, cuts)
        tm.engine.end_sequences(s)
        assert_close(got, ref, dtype, f"{name} {what}")
    tm.engine.check_kernels()
    tm.engine.cache.check()


@pytest.mark.parametrize("name,dtype", [("R", "float32"), ("R", "bfloat16"), ("P", "float32")])
def test_a_long_prompt_takes_the_chunked_kernels(name, dtype):
    """600 tokens in one step (the recurrences' passes over chunks, the many-token projection kernels)
    against the same tokens in portions and one by one."""
    tm = BModel(name, dtype, seed=17, max_tokens=2048)
    toks = tokens_of(np.random.default_rng(23), 600, tm.cfg["vocab"])
    ref = tm.reference(toks)
    for cuts in ([600], [300, 280], [257, 256, 64]):
        s = tm.engine.start_sequences(1)
        got = _feed(tm, s[0], toks, cuts)
        tm.engine.end_sequences(s)
        assert_close(got, ref, dtype, f"{name} cut as {cuts}")


@pytest.mark.parametrize("name,dtype", BOTH)
def test_unequal_batches_equal_each_request_alone(name, dtype):
    tm = BModel(name, dtype, seed=5, max_tokens=1024)
    rng = np.random.default_rng(2)
    V = tm.cfg["vocab"]
    lens, pre = [1, 37, 141, 66], [1, 20, 100, 64]
    reqs = [tokens_of(rng, n, V) for n in lens]
    slots = tm.engine.start_sequences(4)
    out = tm.step_np(slots, [r[:p] for r, p in zip(reqs, pre)], "all")
    got, at = [], 0
    for p in pre:
        got.append([out[at:at + p]])
        at += p
    fed, live = list(pre), [i for i in range(4) if pre[i] < lens[i]]
    tm.engine.end_sequences([slots[i] for i in range(4) if pre[i] >= lens[i]])
    while live:
        out = tm.step_np([slots[i] for i in live], [[reqs[i][fed[i]]] for i in live], "last")
        for j, i in enumerate(live):
            got[i].append(out[j:j + 1])
            fed[i] += 1
        done = [i for i in live if fed[i] >= lens[i]]
        tm.engine.end_sequences([slots[i] for i in done])      # shorter requests end earlier
        live = [i for i in live if i not in done]
    if dtype == "float32":
        for i, r in enumerate(reqs):
            assert_close(np.concatenate(got[i]), tm.reference(r), dtype, f"{name} request {i} of the batch")
    else:
        assert_close(np.concatenate([np.concatenate(g) for g in got]), np.concatenate([tm.reference(r) for r in reqs]),
                     dtype, f"{name} all requests of the batch")
    assert tm.engine.cache.slots.held_count == 0
    tm.engine.cache.check()


@pytest.mark.parametrize("name,dtype", [("P", "float32"), ("R", "bfloat16"), ("Q", "float32")])
def test_slots_pages_and_state_are_clean_when_used_again(name, dtype):
    """A cache that holds one request at a time: every request gets the slot, the pages, the recurrent
    states and the kept convolution inputs that the one before left behind."""
    tm = BModel(name, dtype, seed=8, max_tokens=192, max_batch=1)
    rng = np.random.default_rng(9)
    for n, cuts in ((170, [100]), (130, [130]), (150, [3, 90]), (5, [])):
        toks = tokens_of(rng, n, tm.cfg["vocab"])
        s = tm.engine.start_sequences(1)
        assert s == [0]
        got = _feed(tm, s[0], toks, cuts)
        tm.engine.end_sequences(s)
        assert_close(got, tm.reference(toks), dtype, f"{name} request of {n} tokens in a used slot")
        tm.engine.cache.check()
    toks = tokens_of(rng, 90, tm.cfg["vocab"])
    s = tm.engine.start_sequences(1)
    _feed(tm, s[0], tokens_of(rng, 70, tm.cfg["vocab"]), [70])
    tm.engine.reset(s[0])
    assert_close(_feed(tm, s[0], toks, [50]), tm.reference(toks), dtype, f"{name} after reset")
    tm.engine.end_sequences(s)


@pytest.mark.parametrize("name", ["P", "Q"])
def test_long_decoding(name):
    """400 tokens one by one: the recurrent states and the windows run far past every edge, and the decode
    steps are replayed from recorded graphs."""
    tm = BModel(name, "float32", seed=13)
    rng = np.random.default_rng(5)
    reqs = [tokens_of(rng, n, tm.cfg["vocab"]) for n in (400, 333)]
    slots = tm.engine.start_sequences(2)
    got = [[], []]
    for t in range(400):
        live = [i for i in (0, 1) if t < len(reqs[i])]
        out = tm.step_np([slots[i] for i in live], [[reqs[i][t]] for i in live], "last")
        for j, i in enumerate(live):
            got[i].append(out[j])
    tm.engine.end_sequences(slots)
    assert len(tm.engine._graphs) > 0, "no decode step was replayed from a graph"
    for i in (0, 1):
        assert_close(np.stack(got[i]), tm.reference(reqs[i]), "float32", f"{name} sequence {i}")


@pytest.mark.parametrize("name", ["P", "R"])
def test_greedy_generation_through_the_entry_point(name):
    tm = BModel(name, "float32", seed=21, max_tokens=512)
    rng = np.random.default_rng(4)
    prompts = [tokens_of(rng, n, tm.cfg["vocab"]) for n in (1, 19, 70)]
    res = tm.model.generate(prompts, max_tokens=14, temperature=0.0, stop_ids=())
    for p, r in zip(prompts, res):
        seq, want = list(p), []
        for _ in range(14):
            want.append(int(np.argmax(tm.reference(seq)[-1])))
            seq.append(want[-1])
        assert r.tokens == want, f"prompt of {len(p)} tokens"
    assert tm.engine.steps_advanced_on_device > 0, "the decode steps were not fed from the device"
    assert tm.engine.cache.slots.held_count == 0


@pytest.mark.parametrize("name", ["P", "Q", "R"])
def test_layers_one_by_one(name):
    """The stream after every layer (32-bit), so that a wrong layer is named."""
    tm = BModel(name, "float32", seed=6)
    toks = tokens_of(np.random.default_rng(1), 45, tm.cfg["vocab"])
    seen = []
    for b in tm.engine.model.blocks:
        def wrap(x, batch, *a, f=b.forward, **k):
            r = f(x, batch, *a, **k)
            seen.append(x.cpu().numpy().copy())
            return r
        b.forward = wrap
    s = tm.engine.start_sequences(1)
    tm.step_np(s, [toks], "last")
    ref = []
    plain.forward(tm.cfg, tm.weights, toks, streams_out=ref)
    assert len(seen) == len(ref)
    for i, (a, r) in enumerate(zip(seen, ref)):
        assert np.abs(a - r).max() <= 1e-4 * max(1.0, np.abs(r).max()), \
            f"layer {i} ({tm.cfg['layers'][i]['type']}): {np.abs(a - r).max():.3e}"


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_configurations_drawn_at_random(seed):
    cfg = random_config(seed)
    tm = BModel(cfg, "float32", seed=seed)
    rng = np.random.default_rng(seed)
    V = cfg["vocab"]
    toks = tokens_of(rng, 140, V)
    ref = tm.reference(toks)
    for cuts in ([140], [100], [2, 67, 3]):
        s = tm.engine.start_sequences(1)
        assert_close(_feed(tm, s[0], toks, cuts), ref, "float32", f"seed {seed} cut as {cuts}")
        tm.engine.end_sequences(s)
    reqs = [tokens_of(rng, n, V) for n in (9, 80, 33)]
    slots = tm.engine.start_sequences(3)
    out = tm.step_np(slots, reqs, "all")
    at = 0
    for r in reqs:
        assert_close(out[at:at + len(r)], tm.reference(r), "float32", f"seed {seed} batch")
        at += len(r)
    tm.engine.end_sequences(slots)
    tmb = BModel(cfg, "bfloat16", seed=seed)
    s = tmb.engine.start_sequences(1)
    assert_close(_feed(tmb, s[0], toks, [90]), tmb.reference(toks), "bfloat16", f"seed {seed} bfloat16")


def test_a_folder_may_hold_the_second_norm_of_a_layer_without_feed_forward():
    cfg = CONFIGS["P"]
    stored = make_weights(cfg, 4, torch.float32)
    stored["l2.norm2"] = torch.ones(cfg["width"])
    tm = BModel(cfg, "float32", weights=stored)
    toks = tokens_of(np.random.default_rng(0), 30, cfg["vocab"])
    s = tm.engine.start_sequences(1)
    assert_close(tm.step_np(s, [toks], "all"), tm.reference(toks), "float32", "unused norm present")


def test_replay_program_and_command_line(tmp_path):
    from test_trace_run_gpu import collect, run_trace
    cfg = CONFIGS["P"]
    stored = make_weights(cfg, 33, torch.float32)
    w = {k: v.double().numpy() for k, v in stored.items()}
    d = write_folder({**cfg, "vocab_size": cfg["vocab"]}, stored, str(tmp_path))   # the shared helper reads this key
    rng = np.random.default_rng(3)
    reqs = {"a": tokens_of(rng, 70, cfg["vocab"]), "b": tokens_of(rng, 33, cfg["vocab"])}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs["a"][:60], "want": list(range(60))},
                                     {"id": "b", "tokens": reqs["b"][:30], "want": [0, 29]}], "end": []}]
    for t in range(10):
        ent = [{"id": "a", "tokens": [reqs["a"][60 + t]], "want": [0]}]
        if t < 3:
            ent.append({"id": "b", "tokens": [reqs["b"][30 + t]], "want": [0]})
        steps.append({"step": t + 1, "entries": ent, "end": ["b"] if t == 2 else (["a"] if t == 9 else [])})
    got = collect(steps, run_trace(d, "float32", 256, steps))
    for rid, toks in reqs.items():
        ref = plain.forward(cfg, w, toks)
        for pos, row in got[rid].items():
            assert_close(row[None], ref[pos][None], "float32", f"request {rid} position {pos}")
    assert sorted(got["a"]) == list(range(70)) and sorted(got["b"]) == [0, 29, 30, 31, 32]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "torchless"), "--temperature", "0",
                        "--max-tokens", "5", "--dtype", "float32", d, "3 17 200 ; 45"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    for prompt, line in zip(([3, 17, 200], [45]), r.stdout.strip().splitlines()):
        seq = list(prompt)
        for tok in line.split():
            assert int(tok) == int(np.argmax(plain.forward(cfg, w, seq)[-1]))
            seq.append(int(tok))


# ---------------------------------------------------------------------------------------------
# Kernels alone
# ---------------------------------------------------------------------------------------------
def _ops(dtype):
    from torchless_rs_b200.csrc import ops
    return ops.core_ops(dtype)


def _dev(a, dtype=torch.float32):
    return torch.as_tensor(np.asarray(a), dtype=dtype).cuda().contiguous()


def _i32(a):
    return torch.as_tensor(np.asarray(a, dtype=np.int32)).cuda()


def _pieces(n, cuts):
    """(start, count) of the steps that feed n tokens in pieces of `cuts`, the rest one by one."""
    out, at = [], 0
    for c in list(cuts) + [1] * n:
        if at >= n:
            break
        c = min(c, n - at)
        out.append((at, c))
        at += c
    return out


def _np(t):
    return t.float().cpu().numpy().astype(np.float64)


def _close(got, ref, tol, what=""):
    """Within `tol` of the largest reference entry."""
    err = np.abs(np.asarray(got, dtype=np.float64) - ref).max()
    assert err <= tol * max(1e-30, np.abs(ref).max()), f"{what}: {err:.3e} of {np.abs(ref).max():.3e}"


# ---- layer norms ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,H", [(1, 7), (3, 96), (5, 130), (9, 512), (2, 1000), (700, 1024), (3, 2048), (1500, 2048),
                                    (5, 4096), (200, 4096), (3, 8192), (2, 8196), (2, 12001)])
def test_layer_norms(dtype, rows, H):
    """Rows whose mean is far from zero (the deviations are 1/300 of it): a variance taken as the difference of
    two means of squares would be lost.  More rows than blocks, few rows, widths past what registers hold."""
    o = _ops(dtype)
    rng = np.random.default_rng(H)
    x = rng.normal(30, 0.1, (rows + 3, H)).astype(np.float32)
    x[:, 0] += 1.0                                # one entry that stands out in every row
    w, b, w2, b2 = (rng.normal(1, 0.5, H).astype(np.float32) for _ in range(4))
    pick = rng.permutation(rows + 3)[:rows].astype(np.int32)
    out = torch.empty((rows, H), device="cuda", dtype=dtype)
    o.layernorm(_dev(x), _dev(w), _dev(b), 1e-5, out, _i32(pick))
    tol = 3e-5 if dtype == torch.float32 else 5e-3
    f64 = lambda a: np.asarray(a, dtype=np.float64)
    _close(_np(out), plain.layer_norm(f64(x)[pick], f64(w), f64(b), 1e-5), tol, "rows picked")
    o.layernorm(_dev(x[:rows]), _dev(w), _dev(b), 1e-5, out)
    _close(_np(out), plain.layer_norm(f64(x)[:rows], f64(w), f64(b), 1e-5), tol, "rows in order")
    # the closing form: y with a row stride of its own, the stream in place, the next norm
    y = rng.normal(-20, 0.1, (rows, H + 4)).astype(np.float32)
    s = x[:rows].copy()
    want = f64(s) + plain.layer_norm(f64(y)[:, :H], f64(w), f64(b), 1e-4)
    for fused in (True, False):
        st = _dev(s)
        then = (_dev(w2), _dev(b2), 1e-6, out) if fused else ()
        o.layernorm_add_layernorm(_dev(y)[:, :H], _dev(w), _dev(b), 1e-4, st, *then)
        _close(_np(st), want, 4e-6, "stream")     # (the 32-bit mean's last bit is 1e-5 of a deviation here)
        if fused:
            _close(_np(out), plain.layer_norm(want, f64(w2), f64(b2), 1e-6), 1e-4 if dtype == torch.float32 else 5e-3, "next")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["rmsnorm", "layernorm"])
def test_a_block_with_scaled_sublayers_takes_either_norm(dtype, kind):
    """x + s * N_b(sub(N(x))) for a sublayer that returns what it is given."""
    from torchless_rs_b200.config import PartSpec
    from torchless_rs_b200.parts import Runtime, lookup
    rt = Runtime("cuda:0", dtype)
    W, T, eps = 72, 19, 1e-5
    rng = np.random.default_rng(3)
    spec = PartSpec(kind, {"size": W, "eps": eps, "bare_name": True})
    names = {"mixer_norm": "n1", "mixer_out_norm": "n1b", "feed_forward_norm": "n2", "feed_forward_out_norm": "n2b"}
    weights = {"p.s1": torch.tensor(rng.normal(1, 0.5, W), dtype=torch.float32),
               "p.s2": torch.tensor(rng.normal(1, 0.5, W), dtype=torch.float32)}
    norms = {}
    for role, n in names.items():
        weights[n] = torch.tensor(rng.normal(1, 0.3, W), dtype=torch.float32)
        weights[n + ".b"] = torch.tensor(rng.normal(0, 0.3, W), dtype=torch.float32)
        norms[role] = lookup("norm", kind)(spec, n, rt)
        norms[role].load(weights)

    class Echo:
        can_overwrite = True

        def __init__(self, f):
            self.f = f

        def forward(self, xn, y, batch, overwrite=False):
            y.copy_(xn.float() * self.f)
    block = lookup("block", "sandwich")(PartSpec("sandwich", {"prefix": "p", "size": W, "scales": ("s1", "s2")}), rt,
                                        Echo(3.0), Echo(-0.5), norms)
    block.load(weights)
    x0 = rng.normal(0, 2, (T, W)).astype(np.float32)
    x = _dev(x0)
    block.forward(x, None)
    g = lambda n: weights[n].double().numpy()

    def norm(u, n):
        if kind == "layernorm":
            return plain.layer_norm(u, g(n), g(n + ".b"), eps)
        return plain.rms_norm(u, g(n), eps)
    ref = x0.astype(np.float64)
    ref = ref + g("p.s1") * norm(3.0 * norm(ref, "n1"), "n1b")
    ref = ref + g("p.s2") * norm(-0.5 * norm(ref, "n2"), "n2b")
    _close(_np(x), ref, 1e-5 if dtype == torch.float32 else 1e-2)


# ---- rotation with an amplitude, values of several layers mixed ------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,G,dim,vdim,rot", [(5, 4, 2, 20, 7, 12), (40, 3, 3, 64, 48, 64), (300, 4, 1, 64, 32, 32),
                                                (300, 6, 2, 20, 12, 20), (270, 2, 2, 16, 16, 0), (333, 8, 2, 128, 128, 128)])
def test_rotation_with_amplitude_and_mixed_values(dtype, T, H, G, dim, vdim, rot):
    """Every form of the kernel (few tokens; many, with and without vector loads): queries and keys turned and
    scaled, the entries past the rotated ones as they were, values left for later layers, values mixed with what
    is there."""
    o = _ops(dtype)
    rng = np.random.default_rng(T + dim)
    cols = (H + G) * dim + G * vdim
    f, amp = plain.frequencies(rotation(rot, 500.0, ramp(6.0, 128, 8.0, 1.0)), rot) if rot else (np.zeros(0), 1.0)
    z = rng.normal(size=(T, cols)).astype(np.float32)
    z64 = z.astype(np.float64)
    pos = np.arange(5, 5 + T)
    n_pages = (5 + T + 63) // 64
    first = rng.normal(size=(T, G * vdim)).astype(np.float32)
    turned = lambda v: plain.rotate_halves(v, pos.astype(np.float64), f, amp)
    q = turned(z64[:, :H * dim].reshape(T, H, dim))
    k = turned(z64[:, H * dim:(H + G) * dim].reshape(T, G, dim))
    v = z64[:, (H + G) * dim:]
    tol = 2e-5 if dtype == torch.float32 else 5e-3
    perm = rng.permutation(n_pages)
    for mix in (None, "first", 0.3, 1.0):
        kp = torch.zeros((n_pages, G, 64, dim), device="cuda", dtype=dtype)
        vp = torch.zeros((n_pages, G, vdim, 64), device="cuda", dtype=dtype)
        qo = torch.zeros((T, H * dim), device="cuda", dtype=dtype)
        fv = _dev(first) if mix is not None else None
        o.rotary_cache_write(_dev(z), _dev(f) if rot else None, rot, 0, False, 1e-5, qo, kp, vp, _i32(pos), _i32(np.zeros(T)),
                             _i32([1]), _i32(np.stack([perm * 0 - 1, perm])), H, G, G, dim, vdim, amplitude=amp,
                             first_values=fv, mix=mix if isinstance(mix, float) else None)
        want_v = plain.mix_values(v, first.astype(np.float64), mix) if isinstance(mix, float) else v
        _close(_np(qo).reshape(T, H, dim), q, tol, f"q {mix}")
        page, at = perm[pos // 64], pos % 64
        _close(_np(kp)[page, :, at], k, tol, f"k {mix}")
        _close(_np(vp)[page, :, :, at].reshape(T, G * vdim), want_v, tol, f"v {mix}")
        if mix is not None:
            _close(_np(fv), v if mix == "first" else first.astype(np.float64), 1e-6, f"first layer's values {mix}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dim,vdim,window,n", [(4, 2, 64, 64, 70, 200), (8, 1, 32, 48, 64, 150), (3, 3, 20, 12, 33, 140),
                                                   (4, 1, 128, 128, 100, 320), (4, 2, 64, 64, None, 300)])
def test_window_edges_through_the_mixer(dtype, H, G, dim, vdim, window, n):
    """One key per case stands out for one query (its score is some ten above the others, rotation and amplitude
    included): just inside the window, just outside, the query itself, the first token; in a prompt, in a
    second portion and in decode steps."""
    o = _ops(dtype)
    from torchless_rs_b200.csrc.attention_bf16 import FAST_HEAD_DIMS, AttentionBf16
    from torchless_rs_b200.parts.runtime import Workspace
    from torchless_rs_b200.parts.sink_attention import run_attention
    rng = np.random.default_rng(dim + n)
    f, amp = plain.frequencies(rotation(dim, 500.0, ramp(6.0, 64, 8.0, 1.0)), dim)
    scale = dim ** -0.5
    z = rng.normal(0, 0.5, (n, (H + G) * dim + G * vdim))
    u = rng.normal(size=dim)
    u *= np.sqrt(14.0 / (scale * amp * amp)) / np.linalg.norm(u)
    back = lambda v, p: plain.rotate_halves(v[None], np.array([-float(p)]), f, 1.0)[0]     # so that rotation undoes it
    w = window or 10 ** 6
    probes = []
    for i in (n - 1, n - 40, 130):
        for j in (i - w + 1, i - w, i, 0, i - 1):
            if 0 <= j <= i and i < n:
                probes.append((i, j))
    fast = AttentionBf16.get(dim) if dtype == torch.bfloat16 and dim == vdim and dim in FAST_HEAD_DIMS else None
    ws, n_pages = Workspace(torch.device("cuda")), (n + 63) // 64
    for i, j in probes:
        zz = z.copy()
        for h in range(H):
            zz[i, h * dim:(h + 1) * dim] = back(u, i)
        for g in range(G):
            zz[j, (H + g) * dim:(H + g + 1) * dim] = back(u, j)
        zz = zz.astype(np.float32).astype(np.float64)
        pos = np.arange(n, dtype=np.float64)
        q = plain.rotate_halves(zz[:, :H * dim].reshape(n, H, dim), pos, f, amp)
        k = plain.rotate_halves(zz[:, H * dim:(H + G) * dim].reshape(n, G, dim), pos, f, amp)
        v = zz[:, (H + G) * dim:].reshape(n, G, vdim)
        mask = plain.visible(n, window)
        ref = np.stack([plain.softmax(q[:, h] @ k[:, h // (H // G)].T * scale, mask) @ v[:, h // (H // G)] for h in range(H)], 1)
        perm = rng.permutation(n_pages)
        for cuts in ([n], [i], [128, 2]):
            kp = torch.zeros((n_pages, G, 64, dim), device="cuda", dtype=dtype)
            vp = torch.zeros((n_pages, G, vdim, 64), device="cuda", dtype=dtype)
            table = _i32(perm[None])
            for at, c in _pieces(n, cuts):
                qo = torch.empty((c, H * dim), device="cuda", dtype=dtype)
                out = torch.empty((c, H * vdim), device="cuda", dtype=dtype)
                tp, ts, sl = _i32(np.arange(at, at + c)), _i32(np.zeros(c)), _i32([0])
                o.rotary_cache_write(_dev(zz[at:at + c]), _dev(f), dim, 0, False, 1e-5, qo, kp, vp, tp, ts, sl, table, H, G, G,
                                     dim, vdim, amplitude=amp)
                if not at <= i < at + c:
                    continue

                class B:
                    n_seqs, is_decode, len_bucket, max_len, max_new = 1, c == 1, 512, at + c, c
                    seq_start, seq_len, seq_slot, new_lens = _i32([0, c]), _i32([at + c]), sl, [at + c]

                class C:
                    k_pages, v_pages, page_table = kp, vp, table
                if fast is None or not fast.run(qo, C, out, B, H, G, window, scale, ws):
                    run_attention(o, qo, kp, vp, None, None, out, tp, ts, sl, table, H, G, dim, vdim, window, 0, scale, None, B, ws)
                got = _np(out)[i - at].reshape(H, vdim)
                _close(got, ref[i], 5e-5 if dtype == torch.float32 else 2e-2, f"query {i}, key {j}, cut {cuts}")
                break


# ---- latent attention ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dim,rot,vdim,rank,n", [(4, 16, 8, 12, 24, 140), (3, 32, 16, 20, 64, 300), (20, 16, 16, 16, 48, 150),
                                                   (2, 24, 0, 8, 33, 90), (5, 64, 32, 64, 128, 200)])
def test_latent_attention_alone(dtype, H, dim, rot, vdim, rank, n):
    """The mixer's part with weights made so that a far key stands out: one token's latent is what one query, far
    behind it, looks for.  A whole step, portions, one token at a time, in permuted pages."""
    from torchless_rs_b200.config import PartSpec
    from torchless_rs_b200.parts import Runtime, lookup
    W = 40
    rng = np.random.default_rng(rank)
    rt = Runtime("cuda:0", dtype)
    scaling = ramp(5.0, 64, 8.0, 1.0)
    p = {"heads": H, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": float((dim + rot) ** -0.5)}
    if rot:
        p["rot"] = rotation(rot, 1000.0, scaling)
    sd = W ** -0.5
    w = {"q": rng.normal(0, sd, (H * (dim + rot), W)), "dkv": rng.normal(0, sd, (rank + rot, W)),
         "dkv.norm": rng.normal(1, 0.2, rank), "uk": rng.normal(0, rank ** -0.5, (H * dim, rank)),
         "uv": rng.normal(0, rank ** -0.5, (H * vdim, rank)), "g": rng.normal(0, sd, (H, W)),
         "o": rng.normal(0, (H * vdim) ** -0.5, (W, H * vdim))}
    store = {k: torch.tensor(v, dtype=torch.float32).to(dtype) for k, v in w.items()}
    w64 = {k: v.double().numpy() for k, v in store.items()}
    h = rng.normal(size=(n, W))
    for i, j in ((n - 1, 1), (n - 2, 64), (70, 0)):        # scale up a query and turn it towards one key
        keys = w64["uk"].reshape(H, dim, rank) @ plain.rms_norm(h[j] @ w64["dkv"].T[:, :rank], w64["dkv.norm"], 1e-5)
        qm = w64["q"].reshape(H, dim + rot, W)[:, :dim]
        pull = np.einsum("hd,hdw->w", keys, qm)
        h[i] = 0.3 * h[i] + 6.0 * pull / np.linalg.norm(pull)
    h = torch.tensor(h, dtype=torch.float32).to(dtype).double().numpy()
    ref = plain.latent_attention(h, w64, p, 1e-5, {})
    spec = PartSpec("latent_attention", {"hidden_size": W, **{k: v for k, v in p.items() if k != "rot"}, "q_rank": None,
                                         "window": None, "eps": 1e-5, "rot_dims": rot, "gate": "head", "sink": False})
    pos = lookup("position", "rope_half_split")(PartSpec("rope_half_split", {
        "head_dim": rot, "theta": 1000.0, "scaling": {"kind": "ramp", **scaling}}), rt) if rot else None
    mixer = lookup("mixer", "latent_attention")(spec, "m", rt, position=pos)
    mixer.load({f"m.{k}": v for k, v in store.items()})
    n_pages = (n + 63) // 64
    perm = rng.permutation(n_pages)

    class Cache:
        pages = torch.zeros((n_pages, 64, rank + rot), device="cuda", dtype=dtype)
        page_table = _i32(np.stack([perm * 0 - 1, perm]))
    for cuts in ([n], [n - 7], [2, 65, 3, 20], [17] * 6):
        Cache.pages.zero_()
        mixer.bind_cache(Cache)
        got = []
        for at, c in _pieces(n, cuts):
            class B:
                token_pos, token_seq, seq_slot, len_bucket = _i32(np.arange(at, at + c)), _i32(np.zeros(c)), _i32([1]), 512
            y = torch.zeros((c, W), device="cuda")
            mixer.forward(_dev(h[at:at + c], dtype), y, B)
            got.append(_np(y))
        _close(np.concatenate(got), ref, 3e-5 if dtype == torch.float32 else 3e-2, f"cut {cuts}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,heads,N,K", [(1, 3, 20, 24), (8, 5, 64, 128), (16, 2, 24, 40), (16, 4, 16, 512), (9, 3, 10, 264),
                                         (17, 2, 48, 96), (130, 3, 80, 64), (64, 2, 128, 512), (5, 2, 7, 33)])
def test_per_head_products_with_gates_per_head(dtype, M, heads, N, K):
    o = _ops(dtype)
    rng = np.random.default_rng(M + N)
    lda = heads * (K + 8) + 4
    a = torch.tensor(rng.normal(size=(M, lda)), dtype=torch.float32)
    w = torch.tensor(rng.normal(size=(heads, N, K)), dtype=torch.float32).to(dtype)
    gate = torch.tensor(rng.normal(0, 2, (M, heads + 3)), dtype=torch.float32)
    ref = np.stack([a.double().numpy()[:, h * (K + 8):h * (K + 8) + K] @ w[h].double().numpy().T for h in range(heads)], 1)
    tol = 1e-5 if dtype == torch.float32 else 1e-2       # the tensor-core kernels round A to bfloat16
    c32 = torch.full((M, heads * (N + 2)), 9.0, device="cuda")
    o.headwise_gemm(a.cuda(), K + 8, w.cuda(), c32, N + 2)
    got = _np(c32).reshape(M, heads, N + 2)
    _close(got[:, :, :N], ref, tol, "32-bit result")
    assert (got[:, :, N:] == 9.0).all()
    c = torch.empty((M, heads * N), device="cuda", dtype=dtype)
    o.headwise_gemm(a.cuda(), K + 8, w.cuda(), c, N, gate=gate.cuda()[:, 2:2 + heads])
    _close(_np(c).reshape(M, heads, N), ref * plain.sigmoid(gate.double().numpy()[:, 2:2 + heads])[:, :, None], tol, "gate per head")


# ---- the selective scan ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("channels", [36, 130])
def test_convolution_with_kept_inputs(dtype, taps, channels):
    """Two sequences side by side in pieces of every size down to one: the inputs ahead of a piece come from what
    was kept, and from zeros at a sequence's start; other slots stay as they are."""
    o = _ops(dtype)
    rng = np.random.default_rng(taps)
    n, col = 50, 4
    z = [torch.tensor(rng.normal(size=(n, col + channels)), dtype=torch.float32).to(dtype) for _ in range(2)]
    w, b = rng.normal(size=(channels, taps)).astype(np.float32), rng.normal(size=channels).astype(np.float32)
    want = [plain.silu(plain.short_convolution(x.double().numpy()[:, col:], w.astype(np.float64), b.astype(np.float64))) for x in z]
    for cuts in ([n], [1, 1, 1, 2, 2, 3, 16, 17], [16, 32, 2], [40]):
        kept = torch.full((4, max(taps - 1, 1), channels), 7.0, device="cuda")
        kept[1:3] = 0.0
        for at, c in _pieces(n, cuts):
            out = torch.empty((2 * c, channels), device="cuda", dtype=dtype)
            o.conv_silu(torch.cat([z[0][at:at + c], z[1][at:at + c]]).cuda(), col, _dev(w), _dev(b), kept, out, _i32([0, c, 2 * c]),
                        _i32([2, 1]))
            for k in (0, 1):
                _close(_np(out)[k * c:k * c + c], want[k][at:at + c], 1e-5 if dtype == torch.float32 else 8e-3, (cuts, at, k))
        if taps > 1:
            for k, slot in ((0, 2), (1, 1)):
                assert np.allclose(_np(kept[slot]), z[k].double().numpy()[n - taps + 1:, col:], atol=1e-6)
            assert (kept[0] == 7.0).all() and (kept[3] == 7.0).all(), "a slot that is not in the step was written"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,N", [(40, 1), (36, 4), (50, 3), (128, 8), (33, 12), (132, 16), (96, 20), (64, 32), (44, 48), (20, 64),
                                 (24, 100), (12, 128), (10, 200), (8, 256), (6, 300), (8, 512)])
def test_selective_scan_alone(dtype, C, N):
    """Every arrangement of a channel's states over lanes, sizes that fill it and sizes that do not; two unequal
    sequences in one step, in portions and one token at a time.  Some rates are so small that the first token is
    still in the state after all the others, some so large that nothing is."""
    o = _ops(dtype)
    rng = np.random.default_rng(C + N)
    lens = (77, 41)
    A = -np.exp(rng.uniform(np.log(1e-4), np.log(30.0), (C, N)))
    D, dtb = rng.normal(size=C), rng.normal(-1.5, 1.0, C)
    cast = lambda a: torch.tensor(a, dtype=torch.float32).to(dtype)
    col = 8
    xs, zs, bcs, dts = [], [], [], []
    for n in lens:
        x = rng.normal(size=(n, C))
        x[0] *= 30.0
        xs.append(cast(x))
        zs.append(cast(rng.normal(size=(n, C + 4))))
        bcs.append(cast(rng.normal(size=(n, col + 2 * N + 4))))
        dts.append(torch.tensor(rng.normal(size=(n, C)), dtype=torch.float32))
    f32 = lambda a: torch.tensor(a, dtype=torch.float32)
    A, D, dtb = f32(A), f32(D), f32(dtb)
    want, last = [], []
    for x, z, bc, dt in zip(xs, zs, bcs, dts):
        bc = bc.double().numpy()
        y, S = plain.selective_scan(x.double().numpy(), plain.softplus(dt.double().numpy() + dtb.double().numpy()),
                                    A.double().numpy(), bc[:, col:col + N], bc[:, col + N:col + 2 * N], D.double().numpy())
        want.append(y * plain.silu(z.double().numpy()[:, :C]))
        last.append(S)
    for cuts in ([77], [1] * 5 + [2, 3, 30], [16, 16, 9], [17, 40]):
        state = torch.full((4, C, N), 5.0, device="cuda")
        state[1:3] = 0.0
        got = [[], []]
        for at, c in _pieces(lens[0], cuts):
            rows = [(k, min(c, n - at)) for k, n in enumerate(lens) if at < n]
            part = lambda ts: torch.cat([ts[k][at:at + m] for k, m in rows]).cuda()
            T = sum(m for _, m in rows)
            y = torch.empty((T, C), device="cuda", dtype=dtype)
            o.selective_scan(part(xs), part(dts), dtb.cuda(), part(bcs), col, A.cuda(), D.cuda(), part(zs)[:, :C], state, y,
                             _i32(np.concatenate([[0], np.cumsum([m for _, m in rows])])), _i32([(2, 1)[k] for k, _ in rows]))
            off = 0
            for k, m in rows:
                got[k].append(_np(y)[off:off + m])
                off += m
        for k, slot in ((0, 2), (1, 1)):
            _close(np.concatenate(got[k]), want[k], 2e-5 if dtype == torch.float32 else 8e-3, f"sequence {k}, cut {cuts}")
            _close(_np(state[slot]), last[k], 2e-5, f"state {k}, cut {cuts}")
        assert (state[0] == 5.0).all() and (state[3] == 5.0).all(), "a slot that is not in the step was written"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_step_sizes_of_every_magnitude(dtype):
    """softplus from far below zero (e^x) to far above (x), as it comes out of one token's state: S = dt x B."""
    o = _ops(dtype)
    C = 64
    pre = np.linspace(-40, 40, C)
    state = torch.zeros((1, C, 1), device="cuda")
    ones = torch.ones((1, C), device="cuda", dtype=dtype)
    bc = torch.ones((1, 2), device="cuda", dtype=dtype)
    y = torch.empty((1, C), device="cuda", dtype=dtype)
    o.selective_scan(ones, _dev(pre[None]), torch.zeros(C, device="cuda"), bc, 0, -torch.ones((C, 1), device="cuda"),
                     torch.zeros(C, device="cuda"), ones, state, y, _i32([0, 1]), _i32([0]))
    ref = plain.softplus(pre.astype(np.float32).astype(np.float64))
    assert np.abs(_np(state)[0, :, 0] / ref - 1).max() <= 4e-6


def test_the_mixed_values_are_what_is_cached():
    """The second layer's pages hold (1 - l) v + l v_first, from prompts and from decode steps."""
    cfg = {**CONFIGS["P"], "layers": [CONFIGS["P"]["layers"][0], CONFIGS["P"]["layers"][3]]}
    tm = BModel(cfg, "float32", seed=2)
    toks = tokens_of(np.random.default_rng(1), 75, cfg["vocab"])
    s = tm.engine.start_sequences(1)
    _feed(tm, s[0], toks, [60])
    seen = {}
    mix = plain.mix_values

    def recording(v, first, lam):
        seen["v"] = mix(v, first, lam)
        return seen["v"]
    plain.mix_values = recording
    try:
        plain.forward(cfg, tm.weights, toks)
    finally:
        plain.mix_values = mix
    view = tm.engine.cache.view(1)
    table = view.page_table.cpu().numpy()[s[0]]
    for p in range(75 - 16, 75):
        got = view.v_pages[int(table[p // 64]), :, :, p % 64].cpu().numpy()
        assert np.abs(got - seen["v"][p]).max() <= 1e-4, p

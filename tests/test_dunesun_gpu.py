"""The Dunesun decoder in the engine against the plain implementation: whole prompts, prefill against
token-by-token decoding, portions down to two tokens, unequal batches, slots, pages and state used again, long
decoding, greedy generation through the entry point, the replay program and the command line; then each
mechanism's kernels alone on inputs made so that a wrong window edge, a missed far key, a sink left out, a
lost state or a convolution that looks past a sequence's start shows."""
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from dunesun_tiny import CONFIGS, DModel, make_weights, random_config, tokens_of, write_folder
from plain import dunesun_plain as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = [(c, d) for c in ("A", "B", "C") for d in ("float32", "bfloat16")]


def assert_close(got, ref, dtype, what=""):
    """32-bit: per logit 2e-5 of the largest logit + 1e-4 |ref| (a few 1e-6 of rounding at a dozen places per
    layer run).  bfloat16: 2 % of the logits' root mean square over all rows and 10 % of the largest logit for
    any one.  What a mechanism's fault does shows in the 32-bit run and in the kernels alone."""
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
    tm = DModel(name, dtype, seed=0)
    toks = tokens_of(np.random.default_rng(11), 150, tm.cfg["vocab"])
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


@pytest.mark.parametrize("name,dtype", [("C", "float32"), ("C", "bfloat16"), ("A", "bfloat16")])
def test_a_long_prompt_takes_the_chunked_kernels(name, dtype):
    """600 tokens in one step (the recurrence in chunks, the many-token attention kernels) against the same tokens
    in portions that end inside, at and just past a chunk."""
    from torchless_rs_b200.csrc import ops
    tm = DModel(name, dtype, seed=0, max_tokens=2048)
    toks = tokens_of(np.random.default_rng(23), 600, tm.cfg["vocab"])
    ref = tm.reference(toks)
    for cuts in ([600], [300, 280], [129, 127, 128, 200], [257, 256, 64]):
        before = ops.launch_counts()
        s = tm.engine.start_sequences(1)
        got = _feed(tm, s[0], toks, cuts)
        tm.engine.end_sequences(s)
        ran = ops.counts_since(before)
        if dtype == "bfloat16":
            assert ran.get("ssd_chunk_out", 0) > 0, "no step ran in chunks"
            assert name != "C" or ran.get("attn_prefill_tc_sink", 0) > 0, "no prompt ran on the tensor-memory kernel"
        assert_close(got, ref, dtype, f"{name} cut as {cuts}")
    tm.engine.check_kernels()


@pytest.mark.parametrize("name,dtype", BOTH)
def test_unequal_batches_equal_each_request_alone(name, dtype):
    tm = DModel(name, dtype, seed=0, max_tokens=1024)
    rng = np.random.default_rng(2)
    lens, pre = [1, 37, 141, 66], [1, 20, 100, 64]
    reqs = [tokens_of(rng, n, tm.cfg["vocab"]) for n in lens]
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


def test_a_batch_of_long_and_short_prompts_in_chunks():
    """Prompts of 300, 5 and 190 tokens in one step: the chunks of one sequence are not those of its neighbour."""
    tm = DModel("C", "bfloat16", seed=0, max_tokens=2048)
    rng = np.random.default_rng(8)
    reqs = [tokens_of(rng, n, tm.cfg["vocab"]) for n in (300, 5, 190)]
    slots = tm.engine.start_sequences(3)
    out = tm.step_np(slots, reqs, "all")
    assert_close(out, np.concatenate([tm.reference(r) for r in reqs]), "bfloat16", "three prompts in one step")
    nxt = [tokens_of(rng, n, tm.cfg["vocab"]) for n in (1, 1, 1)]
    out = tm.step_np(slots, nxt, "last")
    assert_close(out, np.stack([tm.reference(r + n)[-1] for r, n in zip(reqs, nxt)]), "bfloat16", "the token after")
    tm.engine.end_sequences(slots)


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "bfloat16"), ("B", "float32")])
def test_slots_pages_and_state_are_clean_when_used_again(name, dtype):
    """A cache that holds one request at a time: every request gets the slot, the pages, the recurrent states and
    the kept convolution inputs (of every pass) that the one before left behind."""
    tm = DModel(name, dtype, seed=0, max_tokens=192, max_batch=1)
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


@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding(name):
    """400 tokens one by one: the states and the windows run far past every edge, and the decode steps are
    replayed from recorded graphs."""
    tm = DModel(name, "float32", seed=0)
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


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(name):
    tm = DModel(name, "float32", seed=0, max_tokens=512)
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


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_layers_one_by_one(name):
    """The stream after every layer run (32-bit), so that a wrong layer is named.  What joins the stream before the
    next pass is taken along by the layer's last kernel, so it is taken off again here."""
    tm = DModel(name, "float32", seed=0)
    toks = tokens_of(np.random.default_rng(1), 45, tm.cfg["vocab"])
    seen = []
    for b in tm.engine.model.blocks:
        def wrap(x, batch, *a, f=b.forward, **k):
            r = f(x, batch, *a, **k)
            y = x.clone()
            for part in k.get("addend") or ():
                if part is not None:
                    y -= part
            seen.append(y.cpu().numpy())
            return r
        b.forward = wrap
    s = tm.engine.start_sequences(1)
    tm.step_np(s, [toks], "last")
    ref = []
    plain.forward(tm.cfg, tm.weights, toks, streams_out=ref)
    assert len(seen) == len(ref) == len(tm.engine.spec.order)
    for i, (a, r) in enumerate(zip(seen, ref)):
        kind = tm.cfg["layers"][tm.engine.spec.order[i]]["type"]
        assert np.abs(a - r).max() <= 1e-5 * max(1.0, np.abs(r).max()), f"run {i} ({kind}): {np.abs(a - r).max():.3e}"


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_configurations_drawn_at_random(seed):
    cfg = random_config(seed)
    tm = DModel(cfg, "float32", seed=0)
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
    tmb = DModel(cfg, "bfloat16", seed=0)
    s = tmb.engine.start_sequences(1)
    assert_close(_feed(tmb, s[0], toks, [90]), tmb.reference(toks), "bfloat16", f"seed {seed} bfloat16")


def test_a_sequence_ends_where_the_position_table_ends():
    from torchless_rs_b200.cache.pages import CacheCapacityError
    cfg = {**CONFIGS["B"], "max_positions": 70}
    tm = DModel(cfg, "float32", seed=0, max_tokens=512)
    toks = tokens_of(np.random.default_rng(0), 71, cfg["vocab"])
    s = tm.engine.start_sequences(1)
    assert_close(_feed(tm, s[0], toks[:70], [60]), tm.reference(toks[:70]), "float32", "up to the last row")
    with pytest.raises(CacheCapacityError):
        tm.engine.step(s, [toks[70:]])
    tm.engine.end_sequences(s)


def test_replay_program_and_command_line(tmp_path):
    from test_trace_run_gpu import collect, run_trace
    cfg = CONFIGS["A"]
    stored = make_weights(cfg, 0, torch.float32)
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


def _np(t):
    return t.detach().double().cpu().numpy()


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


# ---- convolution, step sizes, kept inputs -----------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 16])
def test_preparation_at_a_sequences_start_and_across_steps(taps, dtype):
    """Two sequences in one step, in pieces of every size, in slots that held another sequence's inputs before
    (cleared when the slot was taken, as the cache does): nothing looks past a sequence's start or at its neighbour."""
    rng = np.random.default_rng(taps)
    H, ch, n = 3, 150, 75
    col_x, col_dt = 5, 5 + ch + 2
    z = [rng.normal(size=(n, col_dt + H)) for _ in range(2)]
    w, b = rng.normal(size=(ch, taps)), rng.normal(size=ch)
    A, dtb = rng.normal(size=H), rng.normal(size=H) * 3
    o, wd = _ops(dtype), _dev(w)
    bd, na, dbd = _dev(b), _dev(-np.exp(A)), _dev(dtb)
    want = [plain.silu(plain.short_convolution(x[:, col_x:col_x + ch], w, b)) for x in z]
    for cuts in ([n], [1, 1, 1, 2, 2, 3, 16, 17], [16, 32, 2], [40]):
        kept = torch.full((4, max(taps - 1, 1), ch), 7.0, device="cuda")
        kept[2] = 0.0
        kept[1] = 0.0
        for at, c in _pieces(n, cuts):
            c2 = c                                              # both sequences bring the same number
            zz = _dev(np.concatenate([z[0][at:at + c], z[1][at:at + c2]]))
            xbc = torch.empty((c + c2, ch), device="cuda", dtype=dtype)
            dtla = torch.empty((c + c2, H, 2), device="cuda")
            o.ssd_prep(zz, col_x, col_dt, wd, bd, kept, xbc, dtla, na, dbd, _i32([0, c, c + c2]), _i32([2, 1]))
            tol = 1e-5 if dtype == torch.float32 else 8e-3
            for k in (0, 1):
                got = _np(xbc[k * c:k * c + c])
                ref = want[k][at:at + c]
                assert (np.abs(got - ref) <= tol * (1 + np.abs(ref))).all(), (cuts, at, c, k)
                dt = plain.softplus(z[k][at:at + c, col_dt:] + dtb)
                d = _np(dtla[k * c:k * c + c])
                assert np.allclose(d[..., 0], dt, rtol=2e-6, atol=1e-7)
                assert np.allclose(d[..., 1], -np.exp(A) * dt, rtol=4e-6, atol=1e-7)
        if taps > 1:
            assert np.allclose(_np(kept[2]), z[0][n - taps + 1:, col_x:col_x + ch], atol=1e-6)
            assert np.allclose(_np(kept[1]), z[1][n - taps + 1:, col_x:col_x + ch], atol=1e-6)
            assert (kept[0] == 7.0).all() and (kept[3] == 7.0).all(), "a slot that is not in the step was written"


# ---- the recurrence -----------------------------------------------------------------------------------------
SSD_SIZES = [(3, 3, 20, 12), (1, 1, 33, 5), (6, 2, 16, 16), (4, 2, 64, 32), (4, 1, 128, 80), (2, 1, 256, 64), (8, 2, 48, 48),
             (2, 2, 300, 20)]


def _ssd_case(rng, n, H, G, N, P, dtype, spread=True):
    """(xbc, dt, A_log, D) with values that the activation type holds; decays from nearly none to nothing left
    within a token, side by side in a head."""
    xbc = torch.from_numpy(rng.normal(size=(n, H * P + 2 * G * N)) / 2).to(dtype)
    dt = np.exp(rng.normal(-1.0, 1.2, (n, H)))
    if spread:
        dt[rng.random((n, H)) < 0.02] = 25.0            # the state is all but gone after such a token
    A = rng.normal(-2.0, 1.0, H)
    A[0] = 1.2
    return xbc, dt.astype(np.float32), A.astype(np.float32), rng.normal(size=H).astype(np.float32)


def _ssd_plain(xbc, dt, A, D, H, G, N, P, S0=None):
    """y of the plain recurrence and the end state, from S0."""
    n = xbc.shape[0]
    v = _np(xbc)
    x, B, C = v[:, :H * P].reshape(n, H, P), v[:, H * P:H * P + G * N].reshape(n, G, N), v[:, H * P + G * N:].reshape(n, G, N)
    if S0 is None:
        S0 = np.zeros((H, N, P))
    y, S = np.zeros((n, H, P)), S0.copy()
    la = (-np.exp(A.astype(np.float64)).astype(np.float32) * dt).astype(np.float64)
    for t in range(n):
        for h in range(H):
            S[h] = np.exp(la[t, h]) * S[h] + float(dt[t, h]) * np.outer(B[t, h // (H // G)], x[t, h])
            y[t, h] = S[h].T @ C[t, h // (H // G)] + float(D[h]) * x[t, h]
    return y.reshape(n, H * P), S


def _ssd_run(o, xbc, dt, A, D, state, starts, slots, H, G, chunked=None):
    na = -np.exp(A.astype(np.float64)).astype(np.float32)
    dtla = _dev(np.stack([dt, (na * dt).astype(np.float32)], axis=-1))
    P = state.shape[3]
    y = torch.full((xbc.shape[0], H * P), float("nan"), device="cuda")
    o.ssd_scan(xbc.cuda(), dtla, _dev(D), state, y, _i32(starts), _i32(slots), H, G, chunked=chunked)
    return _np(y)


@pytest.mark.parametrize("H,G,N,P", SSD_SIZES)
def test_recurrence_in_32_bit_and_short_steps(H, G, N, P):
    """The walk: two sequences in used slots, in pieces; every piece goes on from the state the one before left."""
    rng = np.random.default_rng(N + P)
    for dtype in (torch.float32, torch.bfloat16):
        o = _ops(dtype)
        for cuts in ([20], [1, 2, 7, 8, 9], []):
            n = 27
            cases = [_ssd_case(rng, n, H, G, N, P, dtype) for _ in range(2)]
            A, D = cases[0][2], cases[0][3]
            state = torch.randn((5, H, N, P), device="cuda")
            state[3] = 0.0
            S1 = _np(state[0])
            got = [[], []]
            for at, c in _pieces(n, cuts):
                xbc = torch.cat([k[0][at:at + c] for k in cases])
                y = _ssd_run(o, xbc, np.concatenate([k[1][at:at + c] for k in cases]), A, D, state, [0, c, 2 * c], [3, 0], H, G,
                             chunked=False)
                got[0].append(y[:c])
                got[1].append(y[c:])
            for k, S0 in ((0, None), (1, S1)):
                ref, S = _ssd_plain(cases[k][0], cases[k][1], A, D, H, G, N, P, S0)
                scale = np.abs(ref).max()
                assert np.abs(np.concatenate(got[k]) - ref).max() <= 4e-6 * scale, (dtype, cuts, k)
                assert np.abs(_np(state[3 if k == 0 else 0]) - S).max() <= 4e-6 * max(1.0, np.abs(S).max())


@pytest.mark.parametrize("H,G,N,P", [s for s in SSD_SIZES if s[2] % 16 == 0 and s[3] % 16 == 0])
def test_recurrence_in_chunks(H, G, N, P):
    """Chunks on the tensor cores against the plain recurrence on the same bfloat16 x, B and C: what the state, the
    decays and the weights lose is held to 1e-4 of the largest output (bfloat16 state or weights would lose 4e-3),
    also where strong decays stand beside weak ones.  Lengths at and around a chunk, unequal sequences, used slots."""
    rng = np.random.default_rng(N * P)
    o = _ops(torch.bfloat16)
    for lens in ([128], [129, 1, 127], [64, 300], [2, 255, 256]):
        cases = [_ssd_case(rng, n, H, G, N, P, torch.bfloat16) for n in lens]
        A, D = cases[0][2], cases[0][3]
        state = torch.randn((len(lens) + 2, H, N, P), device="cuda")
        slots = [len(lens) + 1 - i for i in range(len(lens))]
        S0 = [_np(state[s]) for s in slots]
        other = state[0].clone()
        starts = np.concatenate([[0], np.cumsum(lens)])
        y = _ssd_run(o, torch.cat([c[0] for c in cases]), np.concatenate([c[1] for c in cases]), A, D, state, starts, slots, H,
                     G, chunked=True)
        assert np.isfinite(y).all()
        for i, c in enumerate(cases):
            ref, S = _ssd_plain(c[0], c[1], A, D, H, G, N, P, S0[i])
            err = np.abs(y[starts[i]:starts[i + 1]] - ref).max()
            assert err <= 1e-4 * np.abs(ref).max(), f"lengths {lens}, sequence {i}: {err:.2e} of {np.abs(ref).max():.1f}"
            assert np.abs(_np(state[slots[i]]) - S).max() <= 5e-5 * max(1.0, np.abs(S).max())
        assert torch.equal(state[0], other), "a slot that is not in the step was written"


@pytest.mark.parametrize("chunked", [False, True])
def test_a_value_written_far_back_is_recalled(chunked):
    """One token writes a value with a key of its own, 700 tokens of other keys and hardly any decay later it is
    read; after a token that decays everything it is gone."""
    H, G, N, P, n = 2, 1, 32, 16, 720
    o = _ops(torch.bfloat16)
    x, B, C = np.zeros((n, H, P)), np.zeros((n, G, N)), np.zeros((n, G, N))
    rng = np.random.default_rng(3)
    B[:, :, 1:] = rng.choice([-1.0, 1.0], (n, G, N - 1)) * 0.5
    x[:] = rng.choice([-1.0, 1.0], (n, H, P))
    B[9] = 0.0
    B[9, 0, 0] = 2.0                                   # entry 0 is written by token 9 alone
    x[9] = 4.0
    C[709:, 0, 0] = 1.0                                 # and read by tokens 709 on
    dt = np.full((n, H), 0.25, dtype=np.float32)
    dt[715, :] = 1e5                                    # everything before is gone
    A = np.full(H, np.log(1e-3), dtype=np.float32)
    x[715] = 0.0
    xbc = torch.from_numpy(np.concatenate([x.reshape(n, -1), B.reshape(n, -1), C.reshape(n, -1)], axis=1)).to(torch.bfloat16)
    state = torch.zeros((1, H, N, P), device="cuda")
    y = _ssd_run(o, xbc, dt, A, np.zeros(H, dtype=np.float32), state, [0, n], [0], H, G, chunked=chunked).reshape(n, H, P)
    assert np.allclose(y[709], 0.25 * 2.0 * 4.0 * np.exp(-1e-3 * 0.25 * 700), rtol=1e-4)
    assert np.abs(y[:9]).max() == 0.0 and np.abs(y[715:]).max() < 1e-30


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("inner,parts", [(36, 1), (36, 3), (30, 6), (256, 2), (4096, 1), (4096, 8), (20000, 1)])
def test_gate_then_norm_in_parts(inner, parts, dtype):
    rng = np.random.default_rng(inner)
    T = 5
    y, z, w = rng.normal(size=(T, inner)) * 3, rng.normal(size=(T, inner + 12)) * 2, rng.normal(size=inner)
    y[:, :inner // parts] *= 50.0                       # parts of very different size: each by its own root mean square
    out = torch.empty((T, inner), device="cuda", dtype=dtype)
    _ops(dtype).ssd_gate_norm(_dev(y), _dev(z)[:, :inner], _dev(w), 1e-5, out, parts)
    ref = plain.gated_group_norm(y, z[:, :inner], w, parts, 1e-5)
    tol = 1e-5 if dtype == torch.float32 else 8e-3
    assert (np.abs(_np(out) - ref) <= tol * (0.1 + np.abs(ref))).all()

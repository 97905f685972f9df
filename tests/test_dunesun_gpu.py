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


# ---- query and key norms over the whole projection, cache pages ------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 16, 16), (3, 3, 10, 7), (1, 1, 13, 40), (8, 2, 64, 48), (40, 8, 128, 128)])
def test_norm_over_the_whole_projection_and_cache_write(H, G, dim, vdim, dtype):
    rng = np.random.default_rng(dim)
    PAGE = 64
    for lens, past in (([1, 1, 1], [0, 63, 64]), ([70, 3], [62, 5])):
        T = sum(lens)
        z = rng.normal(size=(T, (H + G) * dim + G * vdim + 8))
        z[:, :dim] *= 20.0                              # one head dominates: a norm per head would show
        qw, kw = rng.normal(size=H * dim), rng.normal(size=G * dim)
        B, per_seq = len(lens), 3
        table = rng.permutation(B * per_seq + 2)[:B * per_seq].reshape(B, per_seq)
        kp = torch.full((B * per_seq + 2, G, PAGE, dim), 9.0, device="cuda", dtype=dtype)
        vp = torch.full((B * per_seq + 2, G, vdim, PAGE), 9.0, device="cuda", dtype=dtype)
        pos = np.concatenate([np.arange(p, p + n) for p, n in zip(past, lens)])
        seq = np.repeat(np.arange(B), lens)
        slot = np.arange(B)[::-1].copy()
        q = torch.empty((T, H * dim), device="cuda", dtype=dtype)
        tab = np.zeros((B, per_seq), dtype=np.int32)
        tab[slot] = table
        _ops(dtype).qk_whole_norm_cache_write(_dev(z), None, _dev(qw), _dev(kw), 1e-6, q, kp, vp, _i32(pos), _i32(seq), _i32(slot),
                                              _i32(tab), H, G, dim, vdim)
        rq = plain.rms_normalise(z[:, :H * dim], 1e-6) * qw
        rk = plain.rms_normalise(z[:, H * dim:(H + G) * dim], 1e-6) * kw
        rv = z[:, (H + G) * dim:(H + G) * dim + G * vdim]
        tol = 1e-5 if dtype == torch.float32 else 8e-3
        assert (np.abs(_np(q) - rq) <= tol * (0.01 + np.abs(rq))).all()
        written = torch.zeros_like(kp[:, 0, :, 0], dtype=torch.bool)
        for t in range(T):
            page, at = table[seq[t], pos[t] // PAGE], pos[t] % PAGE
            written[page, at] = True
            k, v = _np(kp[page, :, at]).reshape(-1), _np(vp[page, :, :, at]).reshape(-1)
            assert (np.abs(k - rk[t]) <= tol * (0.01 + np.abs(rk[t]))).all() and (np.abs(v - rv[t]) <= tol * (0.01 + np.abs(rv[t]))).all()
        assert (kp.permute(0, 2, 1, 3)[~written] == 9.0).all() and (vp.permute(0, 3, 1, 2)[~written] == 9.0).all()


# ---- attention: window edges, far keys, one added to the denominator ----------------------------------------------
class _View:
    def __init__(self, kp, vp, table):
        self.k_pages, self.v_pages, self.page_table = kp, vp, table


class _Step:
    def __init__(self, start, lens, slot, max_new, n, is_decode):
        self.seq_start, self.seq_len, self.seq_slot, self.max_new, self.n_seqs, self.is_decode = start, lens, slot, max_new, n, is_decode
        self.max_len = None


def _attend(dtype, q, kp, vp, table, first, n, H, G, dim, vdim, window, scale, sink, tensor_memory):
    """The queries of positions first .. first + n - 1 of one sequence, by the kernel the step would take."""
    from torchless_rs_b200.csrc.attention_bf16 import AttentionBf16
    from torchless_rs_b200.parts.sink_attention import run_attention
    pos = _i32(np.arange(first, first + n))
    seq, slot, start, lens = _i32([0] * n), _i32([0]), _i32([0, n]), _i32([first + n])
    out = torch.full((n, H * vdim), float("nan"), device="cuda", dtype=dtype)
    step = _Step(start, lens, slot, n, 1, n == 1)
    if tensor_memory:
        assert AttentionBf16.get(dim).run_prompt(q, _View(kp, vp, table), out, step, H, G, window, scale, sink=sink)
    else:
        run_attention(_ops(dtype), q, kp, vp, None, sink, out, pos, seq, slot, table, H, G, dim, vdim, window, 0, scale, None,
                      step)
    return _np(out).reshape(n, H, vdim)


@pytest.mark.parametrize("dtype,H,G,dim,vdim", [(torch.float32, 4, 2, 24, 20), (torch.float32, 2, 1, 64, 300),
                                                (torch.bfloat16, 4, 2, 24, 20), (torch.bfloat16, 4, 4, 32, 48),
                                                (torch.bfloat16, 8, 2, 64, 64), (torch.bfloat16, 4, 1, 128, 128),
                                                (torch.bfloat16, 2, 1, 200, 400)])
@pytest.mark.parametrize("window", [None, 1, 20, 64, 65, 130])
def test_keys_that_stand_out_at_a_windows_edge_and_far_back(dtype, H, G, dim, vdim, window):
    """A key scaled so that its score stands out by tens: just inside the window it decides the output, just outside
    it changes nothing; keys on page borders and hundreds of tokens back; as a decode step, a few tokens and a
    long run (the tensor-memory kernel where it takes the sizes)."""
    from torchless_rs_b200.csrc.attention_bf16 import AttentionBf16
    rng = np.random.default_rng(dim + (window or 0))
    n, PAGE = 330, 64
    scale = 1.0 / np.sqrt(dim)
    k = rng.normal(size=(n, G, dim)) * 0.3
    v = rng.normal(size=(n, G, vdim))
    q = rng.normal(size=(n, H, dim)) * 0.3
    u = np.ones(dim) / np.sqrt(dim)                     # the direction of the pairs that stand out
    loud = [0, 63, 64, 127, 190, 300]
    for j in loud:
        k[j] += 6.0 * np.sqrt(dim) * u * (1 if j % 2 else 0.8)
    q += 1.0 * np.sqrt(dim) ** 0.5 * u
    pages = (n + PAGE - 1) // PAGE
    table = rng.permutation(pages + 1)[:pages]
    kp = torch.zeros((pages + 1, G, PAGE, dim), device="cuda", dtype=dtype)
    vp = torch.zeros((pages + 1, G, vdim, PAGE), device="cuda", dtype=dtype)
    kd, vd, qd = _dev(k, dtype), _dev(v, dtype), _dev(q, dtype)
    for p in range(pages):
        m = min(PAGE, n - p * PAGE)
        kp[table[p], :, :m] = kd[p * PAGE:p * PAGE + m].permute(1, 0, 2)
        vp[table[p], :, :, :m] = vd[p * PAGE:p * PAGE + m].permute(1, 2, 0)
    tab = _i32(table[None])
    # the oracle on the values the kernel gets
    qs, ks, vs = _np(qd), _np(kd), _np(vd)
    mask = plain.visible(n, window)
    ref = np.zeros((n, H, vdim))
    for h in range(H):
        ref[:, h] = plain.softmax_plus_one(qs[:, h] @ ks[:, h // (H // G)].T * scale, mask) @ vs[:, h // (H // G)]
    sink = torch.zeros(H, device="cuda")
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    edges = sorted({min(n - 1, j + d) for j in loud for d in ((window or 1) - 1, window or 1)})
    takes = dtype == torch.bfloat16 and AttentionBf16.takes_prompts(dim, vdim, H // G)
    runs = [(e, 1, False) for e in edges] + [(60, 5, False), (125, 7, False), (0, n, False)]
    if takes:
        runs += [(0, n, True), (64, n - 64, True), (101, 200, True)]
    for first, m, tm in runs:
        got = _attend(dtype, qd[first:first + m].reshape(m, -1).contiguous(), kp, vp, tab, first, m, H, G, dim, vdim, window, scale,
                      sink, tm)
        r = ref[first:first + m]
        assert np.isfinite(got).all()
        bad = np.abs(got - r) > tol * (1.0 + np.abs(r))
        assert not bad.any(), (f"window {window}, queries {first}..{first + m - 1}, tensor memory {tm}: "
                               f"{np.abs(got - r).max():.2e} at {np.argwhere(bad)[0]}")


@pytest.mark.parametrize("dim", [48, 64, 128])
@pytest.mark.parametrize("level", [-40.0, -3.0, 0.0, 3.0, 40.0])
def test_the_added_one_takes_its_share(dim, level):
    """Every score equals `level`: a key's weight is e^level / (1 + n e^level), nearly nothing far below zero, 1 / n far
    above; by every kernel and however many tokens the step brings."""
    from torchless_rs_b200.csrc.attention_bf16 import AttentionBf16
    H, G, n = 4, 2, 200
    k = torch.zeros((4, G, 64, dim), device="cuda", dtype=torch.bfloat16)
    k[:, :, :, 0] = 1.0
    v = torch.ones((4, G, dim, 64), device="cuda", dtype=torch.bfloat16)
    q = torch.zeros((n, H, dim), device="cuda", dtype=torch.bfloat16)
    q[:, :, 0] = level
    tab = _i32([[2, 0, 3, 1]])
    sink = torch.zeros(H, device="cuda")
    seen = np.minimum(np.arange(n) + 1, 90)
    want = 1.0 / (1.0 + np.exp(-level) / seen)
    for first, m, tm in ((0, n, False), (150, 1, False), (7, 3, False)) + (((0, n, True),) if dim % 64 == 0 else ()):
        got = _attend(torch.bfloat16, q[first:first + m].reshape(m, -1).contiguous(), k, v, tab, first, m, H, G, dim, dim, 90, 1.0,
                      sink, tm)
        assert np.allclose(got, want[first:first + m, None, None], rtol=1e-2), (first, m, tm)


# ---- experts and the closing kernel -----------------------------------------------------------------------------
@pytest.mark.parametrize("E,top", [(1, 1), (3, 3), (5, 2), (33, 4), (64, 8), (512, 6)])
def test_choice_by_logits_and_softmax_over_the_chosen(E, top):
    rng = np.random.default_rng(E)
    T = 70
    z, b = rng.normal(size=(T, E + 3)) * 2, rng.normal(size=E) * 2
    z[0], b0 = 0.0, np.zeros(E)                        # all tie: the lower indices
    z[1, :E] = -1e30                                    # far below zero, still a softmax over the chosen
    for bias in (b.astype(np.float32), b0.astype(np.float32), None):
        zz = z.astype(np.float32)
        idx = torch.empty((T, top), dtype=torch.int32, device="cuda")
        wt = torch.empty((T, top), device="cuda")
        _ops(torch.float32).moe_route_chosen(_dev(zz)[:, :E], None if bias is None else _dev(bias), top, idx, wt)
        zb = zz[:, :E] + (0 if bias is None else bias)
        ri, rw = plain.route(zb.astype(np.float64), top)
        assert (idx.cpu().numpy() == ri).all()
        assert np.allclose(_np(wt), rw, rtol=2e-6, atol=1e-7)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,ff,E,top,T", [(96, 40, 6, 2, 50), (82, 33, 3, 2, 7), (256, 128, 8, 3, 200), (128, 64, 4, 4, 1)])
def test_experts_products_and_closing_kernel(W, ff, E, top, T, dtype):
    """Plan, grouped products with silu(gate) * up, and the closing kernel with every combination of its terms,
    against the plain experts; one expert is chosen by nobody, one by every token."""
    rng = np.random.default_rng(W + T)
    o = _ops(dtype)
    rnd = lambda *s: _np(torch.from_numpy(rng.normal(size=s)).to(dtype))
    h, wg, wu, wd = rnd(T, W), rnd(E, ff, W) / W ** 0.5, rnd(E, ff, W) / W ** 0.5, rnd(E, W, ff) / ff ** 0.5
    cast = lambda a: _np(torch.from_numpy(a).to(dtype))
    wg, wu, wd = cast(wg), cast(wu), cast(wd)
    z = rng.normal(size=(T, E))
    if top < E:
        z[:, 1] = -50.0
    z[:, 0] = 50.0
    ri, rw = plain.route(z, top)
    idx, wt = _i32(ri), _dev(rw)
    off = torch.empty(E + 1, dtype=torch.int32, device="cuda")
    row_token = torch.empty(T * top, dtype=torch.int32, device="cuda")
    row_of = torch.empty((T, top), dtype=torch.int32, device="cuda")
    o.moe_plan(idx, E, off, row_token, row_of)
    act = torch.empty((T * top, ff), device="cuda", dtype=dtype)
    yk = torch.empty((T * top, W), device="cuda")
    w_up = _dev(np.concatenate([wg, wu], axis=1), dtype)
    o.moe_gemm(_dev(h, dtype), row_token, w_up, act, off, up=True, act=0)
    o.moe_gemm(act, None, _dev(wd, dtype), yk, off, up=False)
    want = np.zeros((T, W))
    for e in range(E):
        r, k = np.nonzero(ri == e)
        want[r] += rw[r, k][:, None] * ((plain.silu(h[r] @ wg[e].T) * (h[r] @ wu[e].T)) @ wd[e].T)
    x, ys, sg = rng.normal(size=(T, W)), rng.normal(size=(T, W)), rng.normal(size=(T, 5)) * 2
    rows, vec, w = rng.normal(size=(T, W)), rng.normal(size=W), rng.normal(size=W)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    for use in range(32):
        xd = _dev(x)
        ref = x.copy()
        kw = {}
        if use & 1:
            kw["experts"], ref = (yk, row_of, wt), ref + want
        if use & 2:
            kw["shared"], ref = (_dev(ys), _dev(sg)[:, 3] if use & 16 else None), ref + (plain.sigmoid(sg[:, 3:4]) if use & 16 else 1.0) * ys
        if use & 4:
            kw["add_rows"], ref = _dev(rows), ref + rows
        if use & 8:
            kw["add_vec"], ref = _dev(vec), ref + vec
        xn = torch.empty((T, W), device="cuda", dtype=dtype)
        if use % 3:
            kw.update(w_next=_dev(w), eps_next=1e-3, xn=xn)
        o.close_block(xd, **kw)
        assert np.abs(_np(xd) - ref).max() <= tol * 4, use
        if use % 3:
            assert (np.abs(_np(xn) - plain.rms_normalise(ref, 1e-3) * w) <= tol * 4).all(), use


@pytest.mark.parametrize("W,T", [(4096, 3), (4096, 600), (20000, 2), (20003, 2)])
def test_closing_kernel_on_wide_rows(W, T):
    rng = np.random.default_rng(W)
    x, rows, vec, w = rng.normal(size=(T, W)), rng.normal(size=(T, W)), rng.normal(size=W), rng.normal(size=W)
    xd, xn = _dev(x), torch.empty((T, W), device="cuda")
    _ops(torch.float32).close_block(xd, None, None, _dev(rows), _dev(vec), _dev(w), 1e-6, xn)
    ref = x + rows + vec
    assert np.allclose(_np(xd), ref, atol=1e-5) and np.allclose(_np(xn), plain.rms_normalise(ref, 1e-6) * w, atol=2e-5)


def test_embedding_keeps_a_copy_and_adds_the_first_passs_row():
    rng = np.random.default_rng(0)
    V, W, P, T = 30, 37, 16, 9
    tab, pos, vec = rng.normal(size=(V, W)), rng.normal(size=(P, W)), rng.normal(size=W)
    tok, at = rng.integers(0, V, T), rng.integers(0, P, T)
    x, copy = torch.empty((T, W), device="cuda"), torch.empty((T, W), device="cuda")
    o = _ops(torch.float32)
    for with_pos in (True, False):
        o.embed(_i32(tok), _dev(tab), x, scale=0.5, position_table=_dev(pos) if with_pos else None, token_pos=_i32(at), copy=copy,
                add_vec=_dev(vec))
        ref = 0.5 * tab[tok] + (pos[at] if with_pos else 0.0)
        assert np.allclose(_np(copy), ref, atol=1e-6) and np.allclose(_np(x), ref + vec, atol=1e-6)


def test_blocks_that_take_no_addend_work_in_repeated_passes():
    """A pre-norm model whose layers run twice, with what stands before a pass added by a kernel of its own: the
    block before must not have prepared its successor's norm from the stream without it."""
    import dataclasses
    from helpers_gpu import TinyModel
    from tiny import CONFIGS as MISTRAL
    from torchless_rs_b200.config import PassStart
    from torchless_rs_b200.engine.engine import Engine
    tm = TinyModel("A", "float32", seed=3, max_tokens=256)
    spec = tm.engine.spec
    n = len(spec.layers)
    W = spec.hidden_size
    rng = np.random.default_rng(2)
    toks = [int(t) for t in rng.integers(0, MISTRAL["A"]["vocab_size"], 20)]
    new = dataclasses.replace(spec, order=tuple(range(n)) * 2, pass_table_name="steps", pass_rows=2,
                              pass_starts={0: PassStart(0), n: PassStart(1, True)})
    w = {k: torch.from_numpy(np.asarray(v, dtype=np.float32)) for k, v in tm.weights.items()}
    w["steps"] = torch.from_numpy(rng.normal(size=(2, W)).astype(np.float32))
    eng = Engine(new, w, tm.engine.rt, 256, use_graphs=False)
    added = []
    ops = eng.rt.ops
    real = ops.close_block
    def spy(x, *a, **k):
        before = x.clone()
        real(x, *a, **k)
        added.append((x - before).cpu().numpy())
    ops.close_block = spy
    try:
        s = eng.start_sequences(1)
        whole = eng.step(s, [toks], "all").cpu().numpy().copy()
    finally:
        del ops.close_block
    assert len(added) == 1 and np.allclose(added[0], _np(w[spec.embedding_name])[toks] + _np(w["steps"])[1], atol=1e-5)
    s2 = eng.start_sequences(1)
    one = np.concatenate([eng.step(s2, [[t]], "last").cpu().numpy().copy() for t in toks])
    assert np.allclose(whole, one, atol=2e-4 * np.abs(whole).max())

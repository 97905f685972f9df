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

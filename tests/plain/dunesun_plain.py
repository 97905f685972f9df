"""Plain, slow restatement of the Dunesun decoder, for tests only: numpy, whole sequences, no cache, one
function per mechanism, token-by-token loops where the design is a recurrence.  It shares no code with
the package under test.

The design in short.  The stream starts as the token's row plus the position's row.  A layer is a parallel
block, x <- x + mixer(h) + ff(h) with one norm h = N(x), N an RMS norm whose stored weight lies around
zero.  The mixer is softmax attention over a sliding window (queries and keys normed over the whole
projection, no rotation, one added to the softmax's denominator) or a selective state-space recurrence
with one decay per head and token (Mamba-2).  The feed-forward is a mixture of experts whose router
weighs the chosen experts by a softmax over their logits, with a shared expert behind a sigmoid gate.  A
run of layers may be repeated with the same weights: before every pass a row of a table is added, and
before every pass but the first the embedded token is added again.  Arrays are float64 by default, so
this is also the oracle for error budgets."""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms_normalise(x: np.ndarray, eps: float) -> np.ndarray:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def model_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    """The norm of the layers and of the output: the stored weight is what the factor has beyond one."""
    return rms_normalise(x, eps) * (1.0 + w)


# ---- embedding and passes --------------------------------------------------------------------------------

def embed(tokens, table: np.ndarray, positions: np.ndarray) -> np.ndarray:
    n = len(tokens)
    return table[np.asarray(tokens)] + positions[:n]


def run_order(n_layers: int, loop) -> list:
    """[(layer, pass or None)]: pass t stands at the first layer of the repeated run's t-th pass."""
    if not loop:
        return [(i, None) for i in range(n_layers)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, None) for i in range(a)]
    for t in range(times):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n_layers)]


def pass_start(x: np.ndarray, embedded: np.ndarray, table: np.ndarray, t: int) -> np.ndarray:
    return x + (embedded if t > 0 else 0.0) + table[t]


# ---- softmax attention -----------------------------------------------------------------------------------

def visible(n: int, size) -> np.ndarray:
    """[n, n] booleans: query i sees key j iff 0 <= i - j (< size, if a size is given)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    ok = j <= i
    if size:
        ok &= (i - j) < size
    return ok


def softmax_plus_one(scores: np.ndarray, mask: np.ndarray) -> np.ndarray:
    """exp(s_j) / (1 + sum over visible j of exp(s_j))."""
    s = np.where(mask, scores, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(-m))


def window_attention(h: np.ndarray, w: dict, p: dict, eps: float) -> np.ndarray:
    n = h.shape[0]
    H, G, dim, vdim = p["heads"], p["kv_heads"], p["dim"], p["vdim"]
    q = rms_normalise(h @ w["q"].T, eps) * w["q.norm"]          # over all heads at once
    k = rms_normalise(h @ w["k"].T, eps) * w["k.norm"]
    q, k = q.reshape(n, H, dim), k.reshape(n, G, dim)
    v = (h @ w["v"].T).reshape(n, G, vdim)
    mask = visible(n, (p.get("mask") or {}).get("size"))
    out = np.zeros((n, H, vdim), dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        out[:, head] = softmax_plus_one((q[:, head] @ k[:, g].T) * p["scale"], mask) @ v[:, g]
    return out.reshape(n, H * vdim) @ w["o"].T


# ---- state-space recurrence ------------------------------------------------------------------------------

def short_convolution(x: np.ndarray, taps: np.ndarray, bias: np.ndarray) -> np.ndarray:
    """x: [n, channels]; taps: [channels, m], the last column weighing the current token, the one before it
    the previous token and so on; what lies before the sequence's start is zero."""
    n, m = x.shape[0], taps.shape[1]
    y = np.zeros_like(x) + bias
    for t in range(n):
        for j in range(m):
            src = t - (m - 1 - j)
            if src >= 0:
                y[t] += taps[:, j] * x[src]
    return y


def selective_scan(x, B, C, dt, A_log, D) -> np.ndarray:
    """x: [n, H, vdim]; B, C: [n, G, N]; dt: [n, H] (positive step sizes).  Token by token:
    S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x."""
    n, H, vdim = x.shape
    G, N = B.shape[1:]
    y = np.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        S = np.zeros((N, vdim), dtype=x.dtype)
        for t in range(n):
            S = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + D[h] * x[t, h]
    return y


def gated_group_norm(y: np.ndarray, z: np.ndarray, w: np.ndarray, groups: int, eps: float) -> np.ndarray:
    """The gate first, then the norm of each of `groups` equal parts of the row by itself."""
    n, inner = y.shape
    g = (y * silu(z)).reshape(n, groups, inner // groups)
    return rms_normalise(g, eps).reshape(n, inner) * w


def mamba2(h: np.ndarray, w: dict, p: dict, eps: float) -> np.ndarray:
    n = h.shape[0]
    H, vdim, N, G = p["heads"], p["vdim"], p["state"], p["groups"]
    inner = H * vdim
    proj = h @ w["in"].T
    z, rest, dt = proj[:, :inner], proj[:, inner:-H], proj[:, -H:]
    c = silu(short_convolution(rest, w["conv"], w["conv.b"]))
    x = c[:, :inner].reshape(n, H, vdim)
    B = c[:, inner:inner + G * N].reshape(n, G, N)
    C = c[:, inner + G * N:].reshape(n, G, N)
    y = selective_scan(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return gated_group_norm(y.reshape(n, inner), z, w["norm"], p["norm_groups"], eps) @ w["o"].T


# ---- experts ---------------------------------------------------------------------------------------------

def swiglu(h: np.ndarray, w: dict) -> np.ndarray:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z: np.ndarray, top: int):
    """The `top` largest logits of each row (ties: the lower index) and the softmax over those alone."""
    idx = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    chosen = np.take_along_axis(z, idx, axis=-1)
    e = np.exp(chosen - chosen.max(axis=-1, keepdims=True))
    return idx, e / e.sum(axis=-1, keepdims=True)


def experts(h: np.ndarray, w: dict, p: dict) -> np.ndarray:
    idx, wt = route(h @ w["router"].T + w["router.b"], p["router"]["top"])
    out = np.zeros_like(h)
    for e in range(p["router"]["experts"]):
        rows, k = np.nonzero(idx == e)
        if len(rows):
            out[rows] += wt[rows, k][:, None] * swiglu(h[rows], sub(w, f"e{e}"))
    if p.get("shared"):
        out += sigmoid(h @ w["shared.sg"].T) * swiglu(h, sub(w, "shared"))
    return out


# ---- layers and the model --------------------------------------------------------------------------------

def sub(w: dict, prefix: str) -> dict:
    return {k[len(prefix) + 1:]: v for k, v in w.items() if k.startswith(prefix + ".")}


MIXERS = {"mamba2": mamba2, "attention": window_attention}


def forward(config: dict, weights: dict, tokens, dtype=np.float64, streams_out=None) -> np.ndarray:
    """Logits [n, vocab] of one sequence.  `weights`: name -> array.  `streams_out`, a list, receives the
    residual stream after every layer run (a repeated layer counts each time)."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    embedded = embed(tokens, w["embed"], w["pos"])
    x = embedded
    for i, t in run_order(len(config["layers"]), config.get("loop")):
        if t is not None:
            x = pass_start(x, embedded, w["loop.step"], t)
        layer, lw = config["layers"][i], sub(w, f"l{i}")
        h = model_norm(x, lw["norm1"], eps)
        y = MIXERS[layer["type"]](h, sub(lw, "mix"), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + experts(h, sub(lw, "mlp"), layer["mlp"])
        x = x + y
        if streams_out is not None:
            streams_out.append(x.copy())
    return model_norm(x, w["final.norm"], eps) @ w["head"].T * config["logit_scale"]

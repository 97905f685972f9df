"""Plain, slow restatement of the Beralix decoder, for tests only: numpy, whole sequences, no cache, one
function per mechanism, token-by-token loops where the design is a recurrence.  It shares no code with the
package under test.

The design in short.  A layer is two sublayers, each between two layer norms (weight and bias) with one factor
per coordinate on what comes out of the second: x <- x + s1 * N1b(mixer(N1(x))); x <- x + s2 * N2b(ff(N2(x))).
The mixer is one of three:
  * `attention`: softmax attention with grouped key/value heads, queries and keys rotated by position on the
    first entries of every head (half-split pairs, frequencies stretched by a ramp over the pairs, sines and
    cosines times one factor), a sliding window, and values that in every such layer after the first are mixed
    with the first one's of the same token;
  * `latent_attention`: causal softmax attention whose keys and values are rebuilt from a low-rank latent, one
    rotated key part shared by all heads, and a sigmoid gate per head;
  * `mamba1`: a selective scan, one decay per channel, state entry and token, behind a short causal convolution.
The feed-forward is SwiGLU or absent; the logits are softly capped.  Arrays are float64 by default, so this is
also the oracle for error budgets."""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


# ---- norms ---------------------------------------------------------------------------------------------

def layer_norm(x: np.ndarray, w: np.ndarray, b: np.ndarray, eps: float) -> np.ndarray:
    """Over the last axis: the mean taken off, divided by the root of the mean squared deviation plus eps."""
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w + b


def rms_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


# ---- positions -----------------------------------------------------------------------------------------

def frequencies(rot: dict, dims: int):
    """(frequencies, factor): one frequency per rotated pair, and what sines and cosines are multiplied by.
    With `scaling`, pair i keeps its frequency where it turns at least `fast` times over `original`
    positions, has it divided by `factor` where it turns at most `slow` times, and a straight line between."""
    base = float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_that_turns(times):
        return dims * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_that_turns(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(sc["slow"]))), dims - 1)
    out = np.empty_like(f)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp)
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x: np.ndarray, positions: np.ndarray, freq: np.ndarray, factor: float) -> np.ndarray:
    """x: [n, ..., d]; entries i and i + m (i < m = len(freq)) turn by positions * freq[i], both times `factor`;
    the entries from 2 m on stay."""
    out, m = x.copy(), len(freq)
    shape = (len(positions),) + (1,) * (x.ndim - 2)
    for i, fi in enumerate(freq):
        a = (positions * fi).reshape(shape)
        c, s = np.cos(a) * factor, np.sin(a) * factor
        u, v = x[..., i], x[..., i + m]
        out[..., i] = u * c - v * s
        out[..., i + m] = v * c + u * s
    return out


# ---- softmax attention ---------------------------------------------------------------------------------

def visible(n: int, size) -> np.ndarray:
    """[n, n] booleans: query i sees key j iff 0 <= i - j (< size, if a size is given)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    ok = j <= i
    if size:
        ok &= (i - j) < size
    return ok


def softmax(scores: np.ndarray, mask: np.ndarray) -> np.ndarray:
    s = np.where(mask, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def mix_values(v: np.ndarray, first: np.ndarray, lam: float) -> np.ndarray:
    return (1.0 - lam) * v + lam * first


def window_attention(h: np.ndarray, w: dict, p: dict, eps: float, shared: dict) -> np.ndarray:
    """`shared` is the model run's own dictionary: the first layer with mixed values leaves them there."""
    n = h.shape[0]
    H, G, dim, vdim = p["heads"], p["kv_heads"], p["dim"], p.get("vdim") or p["dim"]
    q = (h @ w["q"].T).reshape(n, H, dim)
    k = (h @ w["k"].T).reshape(n, G, dim)
    v = (h @ w["v"].T).reshape(n, G, vdim)
    rot = p.get("rot")
    if rot and rot.get("dims"):
        f, factor = frequencies(rot, int(rot["dims"]))
        pos = np.arange(n, dtype=np.float64)
        q, k = rotate_halves(q, pos, f, factor), rotate_halves(k, pos, f, factor)
    if p.get("v_mix"):
        if "first_values" not in shared:
            shared["first_values"] = v
        else:
            v = mix_values(v, shared["first_values"], float(w["vmix"]))
    mask = visible(n, (p.get("mask") or {}).get("size"))
    out = np.zeros((n, H, vdim))
    for head in range(H):
        g = head // (H // G)
        out[:, head] = softmax((q[:, head] @ k[:, g].T) * p["scale"], mask) @ v[:, g]
    return out.reshape(n, H * vdim) @ w["o"].T


def latent_attention(h: np.ndarray, w: dict, p: dict, eps: float, shared: dict) -> np.ndarray:
    n = h.shape[0]
    H, dim, rd, vdim, rank = p["heads"], p["dim"], p.get("rot_dim") or 0, p.get("vdim") or p["dim"], p["kv_rank"]
    q = (h @ w["q"].T).reshape(n, H, dim + rd)
    dkv = h @ w["dkv"].T
    c, kr, qr = rms_norm(dkv[:, :rank], w["dkv.norm"], eps), dkv[:, rank:], q[:, :, dim:]
    if rd and p.get("rot"):
        f, factor = frequencies(p["rot"], rd)
        pos = np.arange(n, dtype=np.float64)
        kr, qr = rotate_halves(kr, pos, f, factor), rotate_halves(qr, pos, f, factor)
    kp = (c @ w["uk"].T).reshape(n, H, dim)
    v = (c @ w["uv"].T).reshape(n, H, vdim)
    gate = sigmoid(h @ w["g"].T)                                            # [n, H]
    mask = visible(n, None)
    out = np.zeros((n, H, vdim))
    for head in range(H):
        s = (q[:, head, :dim] @ kp[:, head].T + qr[:, head] @ kr.T) * p["scale"]
        out[:, head] = (softmax(s, mask) @ v[:, head]) * gate[:, head:head + 1]
    return out.reshape(n, H * vdim) @ w["o"].T


# ---- selective scan ------------------------------------------------------------------------------------

def short_convolution(x: np.ndarray, taps: np.ndarray, bias: np.ndarray) -> np.ndarray:
    """x: [n, channels]; taps: [channels, m], the last column weighing the current token, the one before
    it the previous token and so on; what lies before the sequence's start is zero."""
    n, m = x.shape[0], taps.shape[1]
    y = np.tile(bias, (n, 1))
    for t in range(n):
        for j in range(m):
            src = t - (m - 1 - j)
            if src >= 0:
                y[t] += taps[:, j] * x[src]
    return y


def selective_scan(x, dt, A, B, C, D, S=None):
    """Token by token.  x, dt: [n, channels]; A: [channels, N]; B, C: [n, N]; D: [channels].  Returns
    (y [n, channels], the state after the last token [channels, N])."""
    S = np.zeros(A.shape) if S is None else S.copy()
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba(h: np.ndarray, w: dict, p: dict, eps: float, shared: dict) -> np.ndarray:
    inner, N, rank = p["inner"], p["state"], p["dt_rank"]
    xz = h @ w["in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(short_convolution(x, w["conv"], w["conv.b"]))
    d = x @ w["x"].T
    dt = softplus(d[:, :rank] @ w["dt"].T + w["dt.b"])
    y, _ = selective_scan(x, dt, -np.exp(w["A_log"]), d[:, rank:rank + N], d[:, rank + N:], w["D"])
    return (y * silu(z)) @ w["o"].T


# ---- layers and the model ------------------------------------------------------------------------------

def sub(w: dict, prefix: str) -> dict:
    return {k[len(prefix) + 1:]: v for k, v in w.items() if k.startswith(prefix + ".")}


MIXERS = {"attention": window_attention, "latent_attention": latent_attention, "mamba1": mamba}


def swiglu(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def soft_cap(z: np.ndarray, cap) -> np.ndarray:
    return cap * np.tanh(z / cap) if cap else z


def forward(config: dict, weights: dict, tokens, dtype=np.float64, streams_out=None) -> np.ndarray:
    """Logits [n, vocab] of one sequence.  `weights`: name -> array.  `streams_out`, a list, receives the
    residual stream after every layer."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)]
    shared: dict = {}
    for i, layer in enumerate(config["layers"]):
        lw = sub(w, f"l{i}")

        def norm(u, name):
            return layer_norm(u, lw[name], lw[name + ".b"], eps)
        y = MIXERS[layer["type"]](norm(x, "norm1"), sub(lw, "mix"), layer["mixer"], eps, shared)
        x = x + norm(y, "norm1b") * lw["ls1"]
        if layer.get("mlp") is not None:
            x = x + norm(swiglu(norm(x, "norm2"), sub(lw, "mlp")), "norm2b") * lw["ls2"]
        if streams_out is not None:
            streams_out.append(x.copy())
    h = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    return soft_cap(h @ w["head"].T, config.get("logit_softcap"))

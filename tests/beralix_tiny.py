"""Small Beralix configurations with weights made here (numpy, not the package's generator), a model folder
written with the `safetensors` package, and a loader through the package's entry point.  Matrices are
N(0, 1/in) so that activations are of order one and attention scores spread over a few units: a key that is
wrongly seen or missed or a lost state changes the result by far more than rounding.

The configurations differ from one another, layer by layer, in every size and in the order of the layers:
heads and key/value heads (equal, one, several per group), key and value sizes that differ and are no multiples
of 4, rotations of all, some or none of a head, with and without stretched frequencies, windows of one key,
inside a page, across pages and absent, values mixed or not (the first layer that mixes in the middle), latents with and without a rotated part, convolutions of one to six taps,
states and channel counts that are no multiples of 4, layers without feed-forward, logits with and without a
cap."""
from __future__ import annotations

import json
import os
import shutil
import tempfile

import numpy as np
import torch

from plain import beralix_plain as plain


def ramp(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def rotation(dims, base=10000.0, scaling=None):
    d = {"dims": dims, "base": base}
    if scaling:
        d["scaling"] = scaling
    return d


def attention(heads, kv_heads, dim, vdim, window, rot, mix, mlp, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "v_mix": mix,
         "scale": scale if scale is not None else 1.0 / float(np.sqrt(dim))}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = rot
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, rot, mlp, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "scale": scale if scale is not None else 1.0 / float(np.sqrt(dim + rot_dim))}
    if rot:
        m["rot"] = rot
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def mamba(inner, state, dt_rank, conv, mlp):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, vocab, layers, eps=1e-5, softcap=None):
    d = {"architecture": "Beralix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}
    if softcap:
        d["logit_softcap"] = softcap
    return d


CONFIGS = {
    # windows inside a page and across one, part of a head rotated, a layer without feed-forward
    "P": config(96, 211, [
        attention(4, 2, 20, 12, 20, rotation(12, 10000.0, ramp(4.0, 64, 8.0, 1.0)), True, dense(120)),
        mamba(40, 6, 5, 4, dense(72)),
        latent(3, 16, 8, 12, 24, rotation(8, 1000.0, ramp(3.0, 128, 16.0, 2.0)), None),
        attention(2, 2, 16, 12, 70, rotation(16, 500.0), True, dense(64)),
    ], softcap=12.0),
    # the recurrence first; sizes that are no multiples of 4; one tap and six; one head; a window of one key, none at
    # all; no rotation; unmixed values ahead of mixed ones; no cap
    "Q": config(82, 130, [
        mamba(30, 33, 13, 1, dense(51)),
        attention(3, 3, 11, 7, None, None, False, dense(33)),
        mamba(27, 3, 1, 6, None),
        attention(4, 1, 14, 10, 1, rotation(6, 100.0), True, dense(30)),
        latent(2, 13, 6, 9, 17, rotation(6, 10000.0), dense(40)),
        attention(5, 1, 8, 10, 33, rotation(8, 10000.0, ramp(2.0, 32, 4.0, 1.0)), True, dense(48)),
        latent(1, 10, 0, 20, 30, None, dense(36)),
    ], eps=3e-6),
    # sizes that the tensor-core kernels take, windows across pages, more than 16 latent heads
    "R": config(320, 520, [
        latent(4, 32, 32, 64, 64, rotation(32, 500000.0, ramp(8.0, 256)), dense(384)),
        attention(8, 2, 64, 64, 130, rotation(64, 500000.0, ramp(4.0, 512)), True, dense(256)),
        mamba(192, 16, 24, 3, dense(320)),
        attention(4, 2, 32, 64, 64, rotation(32, 10000.0), True, dense(256)),
        latent(20, 16, 16, 16, 48, rotation(16, 10000.0), dense(192)),
        mamba(128, 64, 16, 4, dense(192)),
    ], softcap=20.0),
}


def random_config(seed: int) -> dict:
    """Another configuration for every seed: two to six layers of any kind in any order, any sizes."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers, values = [], None        # values: what the layers that mix agree on

    def rot(dims):
        if not dims:
            return None
        sc = ramp(float(pick(1.0, 2.0, 8.0, 40.0)), int(pick(64, 512, 4096)), float(pick(4, 32)), float(pick(1, 2))) \
            if rng.random() < 0.7 else None
        return rotation(dims, float(pick(100.0, 10000.0, 500000.0)), sc)
    for _ in range(int(rng.integers(2, 7))):
        mlp = dense(pick(24, 40, 64, 100)) if rng.random() < 0.85 else None
        kind = pick("a", "a", "l", "m")
        if kind == "a":
            G = pick(1, 2, 4)
            dim = pick(8, 16, 24, 32, 64)
            mix = bool(rng.random() < 0.7)
            vdim = pick(8, 16, 24, 32, 64)
            if mix and values is None:
                values = (G, vdim)
            if mix:
                G, vdim = values
            layers.append(attention(G * pick(1, 2, 4), G, dim, vdim, pick(None, 1, 3, 30, 64, 65, 100),
                                    rot(pick(0, dim // 2, dim)), mix, mlp))
        elif kind == "l":
            rd = pick(0, 4, 8, 16)
            layers.append(latent(pick(1, 3, 4), pick(8, 16, 24), rd, pick(8, 16, 20), pick(16, 20, 32, 64), rot(rd), mlp))
        else:
            layers.append(mamba(pick(24, 32, 50, 96), pick(1, 4, 8, 12, 16, 24), pick(1, 4, 7, 16), pick(1, 2, 3, 4, 5), mlp))
    return config(pick(64, 72, 100, 128), pick(97, 150, 256), layers, eps=pick(1e-6, 1e-5),
                  softcap=pick(None, 5.0, 30.0))


def tensor_shapes(cfg: dict) -> dict:
    """Tensor names and shapes, as the design lays them out."""
    W, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        subs = ("1",) if l.get("mlp") is None else ("1", "2")
        for s in subs:
            for n in (f"norm{s}", f"norm{s}b"):
                out[p + n], out[p + n + ".b"] = (W,), (W,)
            out[p + "ls" + s] = (W,)
        if l["type"] == "attention":
            H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.v": (G * v, W), p + "mix.o": (W, H * v)})
            if m["v_mix"]:
                out[p + "mix.vmix"] = ()
        elif l["type"] == "latent_attention":
            H, d, r, v, k = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            out.update({p + "mix.q": (H * (d + r), W), p + "mix.dkv": (k + r, W), p + "mix.dkv.norm": (k,),
                        p + "mix.uk": (H * d, k), p + "mix.uv": (H * v, k), p + "mix.g": (H, W), p + "mix.o": (W, H * v)})
        else:
            C, N, R, t = m["inner"], m["state"], m["dt_rank"], m["conv"]
            out.update({p + "mix.in": (2 * C, W), p + "mix.conv": (C, t), p + "mix.conv.b": (C,), p + "mix.x": (R + 2 * N, C),
                        p + "mix.dt": (C, R), p + "mix.dt.b": (C,), p + "mix.A_log": (C, N), p + "mix.D": (C,),
                        p + "mix.o": (W, C)})
        if l.get("mlp"):
            f = l["mlp"]["ff"]
            out.update({p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f)})
    out["final.norm"], out["final.norm.b"] = (W,), (W,)
    out["head"] = (cfg["vocab"], W)
    return out


def make_weights(cfg: dict, seed: int, store: torch.dtype) -> dict:
    """name -> torch tensor in `store`."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith(".conv"):
            v = rng.normal(0, 1.0 / np.sqrt(shape[1]), shape) + (np.arange(shape[1]) == shape[1] - 1)
        elif name.endswith(".A_log"):
            v = rng.normal(-0.5, 1.0, shape)
        elif name.endswith(".dt.b"):
            v = rng.normal(-1.5, 1.0, shape)
        elif name.endswith(".vmix"):
            v = rng.uniform(0.2, 0.8)
        elif name.endswith(".b"):
            v = rng.normal(0, 0.3, shape)
        elif len(shape) == 1:
            v = 1.0 + rng.normal(0, 0.2, shape)
        elif name == "embed":
            v = rng.normal(0, 1.0, shape)
        elif name == "head":
            v = rng.normal(0, 3.0 / np.sqrt(shape[1]), shape)      # so that a cap bites
        else:
            v = rng.normal(0, 1.0 / np.sqrt(shape[1]), shape)
        out[name] = torch.from_numpy(np.asarray(v, dtype=np.float32)).to(store)
    return out


def write_folder(cfg: dict, weights: dict, where: str | None = None) -> str:
    from safetensors.torch import save_file
    d = where or tempfile.mkdtemp(prefix="tl_beralix_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


class BModel:
    """A configuration loaded through the package's entry point, with the plain implementation (in
    float64, on the stored values) beside it."""

    def __init__(self, cfg, dtype: str, seed: int = 0, max_tokens: int = 1024, max_batch=None, weights=None):
        import torchless_rs_b200 as tl
        self.cfg = CONFIGS[cfg] if isinstance(cfg, str) else cfg
        store = torch.float32 if dtype == "float32" else torch.bfloat16
        self.stored = weights if weights is not None else make_weights(self.cfg, seed, store)
        self.weights = {k: v.to(torch.float64).numpy() for k, v in self.stored.items()}
        d = write_folder(self.cfg, self.stored)
        try:
            self.model = tl.load(d, dtype=dtype, max_tokens=max_tokens, max_batch=max_batch)
        finally:
            shutil.rmtree(d, ignore_errors=True)
        self.engine = self.model.engine
        self._ref = {}

    def reference(self, tokens) -> np.ndarray:
        key = tuple(tokens)
        if key not in self._ref:
            self._ref[key] = plain.forward(self.cfg, self.weights, list(tokens))
        return self._ref[key]

    def step_np(self, slots, tokens, want) -> np.ndarray:
        return self.engine.step(slots, tokens, want).float().cpu().numpy().copy()


def tokens_of(rng, n, vocab):
    return [int(t) for t in rng.integers(0, vocab, size=n)]

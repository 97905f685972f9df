"""Small Dunesun configurations with weights made here (numpy, not the package's generator), a model folder
written with the `safetensors` package, and a loader through the package's entry point.  Matrices are
N(0, 1/in) so that activations are of order one and attention scores spread over a few units: a key that is
wrongly seen or missed, a sink that is left out or a lost state changes the result by far more than rounding.

A token's choice of experts is a step function of the stream, so two sound computations may differ where two
logits nearly tie.  Here the routers read only the stream's first `TAGS` coordinates, which the embedding sets
to plus or minus a constant and which nothing else writes, and a router is the best of many drawn: the choice
depends on the token, and the logits of the last expert chosen and the first left out stay apart
(`choice_margin` says by how much).

The configurations differ from one another, layer by layer, in every size and in the order of the layers:
heads and key/value heads (equal, one, several per group), key and value sizes that differ and are no
multiples of 4, windows of one key, inside a page, across pages and absent, convolutions of one to six taps,
states that are not square, one group, several, one per head, norms in one and several parts, one expert, all
experts chosen, with and without a shared expert, layers without feed-forward, repeated runs at the start, in
the middle and over all layers, and none."""
from __future__ import annotations

import json
import os
import shutil
import tempfile

import numpy as np
import torch

from plain import dunesun_plain as plain

TAGS = 4


def attention(heads, kv_heads, dim, vdim, window, mlp, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
         "scale": scale if scale is not None else 2.0 / float(np.sqrt(dim))}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mamba(heads, groups, state, vdim, conv, norm_groups, mlp):
    return {"type": "mamba2", "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": mlp}


def moe(ff, experts, top, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def config(width, vocab, layers, loop=None, eps=1e-6, logit_scale=1.0, max_positions=1024):
    d = {"architecture": "Dunesun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale,
         "max_positions": max_positions, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CONFIGS = {
    # windows inside a page and across one; a state the tensor-core kernels do not take; a run in the middle,
    # three times, with a layer without feed-forward in it
    "A": config(96, 211, [
        mamba(3, 3, 20, 12, 4, 3, moe(40, 6, 2, 56)),
        attention(4, 2, 16, 16, 20, moe(64, 3, 1)),
        mamba(4, 2, 16, 16, 2, 1, None),
        attention(3, 1, 24, 16, 70, moe(48, 5, 3, 24)),
    ], loop=(1, 3, 3), logit_scale=0.7),
    # attention first; as many key/value heads as heads; a window of one key, none at all; one tap and six; one head;
    # widths and sizes that are no multiples of 4; one expert; all experts chosen; no repeated run
    "B": config(82, 130, [
        attention(3, 3, 10, 7, 1, moe(30, 1, 1, 18)),
        mamba(1, 1, 33, 5, 6, 1, moe(20, 4, 4)),
        attention(2, 1, 13, 22, None, None),
        mamba(6, 3, 8, 9, 1, 2, moe(33, 3, 2, 33)),
    ], eps=3e-5, logit_scale=1.5),
    # sizes that the tensor-core kernels take, windows across pages; two column tiles of a state; every layer
    # twice
    "C": config(256, 520, [
        attention(8, 2, 64, 64, 130, moe(128, 8, 3, 96)),
        mamba(8, 2, 64, 32, 4, 2, moe(96, 4, 2, 128)),
        mamba(4, 1, 128, 80, 3, 1, moe(64, 5, 2)),
        attention(4, 4, 32, 48, 64, moe(96, 6, 2, 64)),
    ], loop=(0, 4, 2), logit_scale=0.4),
}


def random_config(seed: int) -> dict:
    """Another configuration for every seed: two to five layers of either kind in any order, any sizes."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    n, layers = int(rng.integers(2, 6)), []
    for _ in range(n):
        E = pick(1, 3, 4, 7)
        mlp = moe(pick(24, 40, 64), E, int(rng.integers(1, E + 1)), pick(None, 32, 50)) if rng.random() < 0.85 else None
        if rng.random() < 0.5:
            G = pick(1, 2, 3)
            layers.append(attention(G * pick(1, 2, 4), G, pick(8, 16, 20, 32, 64), pick(8, 16, 24, 32, 64),
                                    pick(None, 1, 3, 30, 64, 65, 100), mlp, scale=float(rng.uniform(0.1, 0.5))))
        else:
            G = pick(1, 2)
            H = G * pick(1, 2, 3)
            P = pick(8, 16, 24, 32, 48)
            layers.append(mamba(H, G, pick(8, 16, 20, 32, 48), P, pick(1, 2, 3, 4, 5), pick(1, 2, H), mlp))
    a = int(rng.integers(0, n))
    loop = (a, int(rng.integers(a + 1, n + 1)), pick(1, 2, 3)) if rng.random() < 0.75 else None
    return config(pick(64, 72, 100, 128), pick(97, 150, 256), layers, loop, eps=pick(1e-6, 1e-5),
                  logit_scale=float(rng.uniform(0.3, 2.0)), max_positions=512)


def tensor_shapes(cfg: dict) -> dict:
    """Tensor names and shapes, as the design lays them out."""
    W, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], W)
    out["pos"] = (cfg["max_positions"], W)
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"] = (W,)
        if l["type"] == "attention":
            H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.v": (G * v, W),
                        p + "mix.q.norm": (H * d,), p + "mix.k.norm": (G * d,), p + "mix.o": (W, H * v)})
        else:
            H, G, N, P, t = m["heads"], m["groups"], m["state"], m["vdim"], m["conv"]
            inner, ch = H * P, H * P + 2 * G * N
            out.update({p + "mix.in": (inner + ch + H, W), p + "mix.conv": (ch, t), p + "mix.conv.b": (ch,),
                        p + "mix.dt_bias": (H,), p + "mix.A_log": (H,), p + "mix.D": (H,), p + "mix.norm": (inner,),
                        p + "mix.o": (W, inner)})
        mlp = l.get("mlp")
        if mlp:
            E, names = mlp["router"]["experts"], []
            out[p + "mlp.router"], out[p + "mlp.router.b"] = (E, W), (E,)
            names = [(f"e{e}", mlp["expert"]["ff"]) for e in range(E)]
            if mlp.get("shared"):
                names.append(("shared", mlp["shared"]["ff"]))
                out[p + "mlp.shared.sg"] = (1, W)
            for n, f in names:
                out.update({p + f"mlp.{n}.gate": (f, W), p + f"mlp.{n}.up": (f, W), p + f"mlp.{n}.down": (W, f)})
    out["final.norm"] = (W,)
    out["head"] = (cfg["vocab"], W)
    return out


def draw_router(rng, width: int, experts: int, top: int):
    """A router over the tag coordinates and its bias whose choice is clear for every pattern of tags and
    every factor that the norm may put on them."""
    tags = np.array([[1.0 - 2.0 * (i >> j & 1) for j in range(TAGS)] for i in range(1 << TAGS)])
    best, best_gap = None, -1.0
    for _ in range(1000):
        r, b = rng.normal(0, 2.0, (experts, TAGS)), rng.normal(0, 0.3, experts)
        z = np.concatenate([f * tags @ r.T + b for f in np.geomspace(0.1, 1.5, 24)])
        s = -np.sort(-z, axis=-1)
        gap = np.inf if top >= experts else (s[:, top - 1] - s[:, top]).min()
        if gap > best_gap:
            best, best_gap = (r, b), gap
        if top >= experts:
            break
    return np.concatenate([best[0], np.zeros((experts, width - TAGS))], axis=1), best[1]


def make_weights(cfg: dict, seed: int, store: torch.dtype) -> dict:
    """name -> torch tensor in `store`."""
    rng = np.random.default_rng(seed)
    out, routers = {}, {}
    for i, l in enumerate(cfg["layers"]):
        if l.get("mlp"):
            r = l["mlp"]["router"]
            routers[f"l{i}.mlp.router"], routers[f"l{i}.mlp.router.b"] = draw_router(rng, cfg["width"], r["experts"], r["top"])
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith(".conv"):
            v = rng.normal(0, 1.0 / np.sqrt(shape[1]), shape) + (np.arange(shape[1]) == shape[1] - 1)
        elif name.endswith(".A_log"):
            v = rng.normal(-1.5, 1.0, shape)
        elif name.endswith(".dt_bias"):
            v = rng.normal(-1.0, 1.0, shape)
        elif name.endswith(("norm1", "final.norm")):
            v = rng.normal(0, 0.2, shape)                    # stored around zero
            if name.endswith("norm1"):
                v[:TAGS] = 0.0
        elif name in routers:
            v = routers[name]
        elif name.endswith(".b"):
            v = rng.normal(0, 0.3, shape)
        elif len(shape) == 1:
            v = 1.0 + rng.normal(0, 0.2, shape)
        elif name == "embed":
            v = rng.normal(0, 1.0, shape)
            v[:, :TAGS] = 2.0 * np.sign(rng.normal(0, 1.0, (shape[0], TAGS)))
        elif name in ("pos", "loop.step"):
            v = rng.normal(0, 0.5, shape)
            v[:, :TAGS] = 0.0
        else:
            v = rng.normal(0, 1.0 / np.sqrt(shape[1]), shape)
            if name.endswith((".mix.o", ".down")):
                v[:TAGS] = 0.0
        out[name] = torch.from_numpy(np.asarray(v, dtype=np.float32)).to(store)
    return out


def choice_margin(cfg: dict, weights: dict, tokens) -> float:
    """The least distance between the logits of the last expert chosen and the first left out, over all
    tokens and layer runs."""
    gaps, route = [np.inf], plain.route

    def recording(z, top):
        if top < z.shape[1]:
            s = -np.sort(-z, axis=-1)
            gaps.append(float((s[:, top - 1] - s[:, top]).min()))
        return route(z, top)
    plain.route = recording
    try:
        plain.forward(cfg, weights, list(tokens))
    finally:
        plain.route = route
    return min(gaps)


def write_folder(cfg: dict, weights: dict, where: str | None = None) -> str:
    from safetensors.torch import save_file
    d = where or tempfile.mkdtemp(prefix="tl_dunesun_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


class DModel:
    """A configuration loaded through the package's entry point, with the plain implementation (in
    float64, on the stored values) beside it."""

    def __init__(self, cfg, dtype: str, seed: int = 0, max_tokens: int = 1024, max_batch=None, weights=None):
        import torchless_rs_b200 as tl
        self.cfg = CONFIGS[cfg] if isinstance(cfg, str) else cfg
        self.dtype = dtype
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
            margin = choice_margin(self.cfg, self.weights, tokens)
            assert margin > (0.03 if self.dtype == "bfloat16" else 1e-3), f"two experts nearly tie ({margin:.1e})"
            self._ref[key] = plain.forward(self.cfg, self.weights, list(tokens))
        return self._ref[key]

    def step_np(self, slots, tokens, want) -> np.ndarray:
        return self.engine.step(slots, tokens, want).float().cpu().numpy().copy()


def tokens_of(rng, n, vocab):
    return [int(t) for t in rng.integers(0, vocab, size=n)]

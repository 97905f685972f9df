"""Typed configuration of the Beralix decoder, read from its config.json.

The design: every sublayer stands between two layer norms with weight and bias, and what comes out of the
second is multiplied coordinate by coordinate (x <- x + s * N_b(sub(N(x)))).  A layer's mixer is one of
  * `attention`: softmax attention with grouped key/value heads, the first `rot.dims` entries of queries and
    keys rotated (pairs (i, i + dims/2); frequencies stretched along a ramp over the pairs, `rot.scaling`), a
    sliding window (`mask.size`), and, with `v_mix`, values that in every such layer after the first are mixed
    with the first one's values of the same token by a learned number;
  * `latent_attention`: causal softmax attention through a low-rank latent, queries straight from the input, a
    rotated key part shared by the heads, and a sigmoid gate per head;
  * `mamba1`: a selective scan over `inner` channels of `state` entries, step sizes through `dt_rank` numbers,
    behind a causal convolution of `conv` taps.
The feed-forward is SwiGLU (`mlp.kind` = "dense") or absent (`mlp` null); the logits are softly capped
(`logit_softcap`).  config.json lists the layers one by one with all their sizes and constants
(`layers[i].type`, `.mixer`, `.mlp`), so layers of one model may differ in all of them.  Tensor names: `embed`,
`l<i>.norm1`, `.norm1b`, `.norm2`, `.norm2b` (each with `.b`), `l<i>.ls1`, `l<i>.ls2`, `l<i>.mix.*`, `l<i>.mlp.*`,
`final.norm`, `final.norm.b`, `head`."""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, Optional, Tuple

from .errors import ConfigError
from .reader import KeyReader
from .spec import LayerSpec, ModelSpec, PartSpec

LAYER_TENSOR_NAMES = {"mixer_norm": "norm1", "mixer_out_norm": "norm1b", "mixer": "mix",
                      "feed_forward_norm": "norm2", "feed_forward_out_norm": "norm2b", "feed_forward": "mlp"}
MIXER_SCALE, FEED_FORWARD_SCALE = "ls1", "ls2"
SWIGLU_NAMES = ("gate", "up", "down")


@dataclass(frozen=True)
class Rotation:
    """Rotary positions of the first `dims` entries, pairs (i, i + dims/2), frequency base^(-2i / dims);
    `scaling` = (factor, original, fast, slow) stretches them along a ramp, None leaves them."""
    base: float
    dims: int
    scaling: Optional[Tuple[float, float, float, float]] = None

    KEYS = ("factor", "original", "fast", "slow")

    @classmethod
    def read(cls, data, where: str, limit: int, exactly: bool = False) -> Optional["Rotation"]:
        if data is None:
            return None
        r = KeyReader(data, where)
        dims = r.integer("dims", limit, minimum=0)
        if dims % 2 or dims > limit:
            raise ConfigError(f"{where}: 'dims' {dims} must be even and at most {limit}")
        if exactly and dims != limit:
            raise ConfigError(f"{where}: 'dims' {dims} must be the rotated part's size {limit}")
        scaling = None
        if data.get("scaling") is not None:
            sr = KeyReader(data["scaling"], f"{where}.scaling")
            scaling = tuple(sr.number(k) for k in cls.KEYS)
        return cls(base=r.number("base"), dims=dims, scaling=scaling) if dims else None

    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = dict(zip(self.KEYS, self.scaling))
        return d

    def part(self) -> PartSpec:
        params: Dict[str, Any] = {"head_dim": self.dims, "theta": self.base}
        if self.scaling is not None:
            params["scaling"] = {"kind": "ramp", **dict(zip(self.KEYS, self.scaling))}
        return PartSpec("rope_half_split", params)


@dataclass(frozen=True)
class WindowAttentionLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    rot: Optional[Rotation]
    v_mix: bool
    mix_role: Optional[str] = None     # "first" or "later" among the layers with mixed values; set by the model

    type = "attention"

    @classmethod
    def read(cls, r: KeyReader) -> "WindowAttentionLayer":
        heads, kv = r.integer("heads"), r.integer("kv_heads")
        if heads % kv:
            raise ConfigError(f"{r.where}: 'heads' {heads} is no multiple of 'kv_heads' {kv}")
        mask = r.data.get("mask")
        window = KeyReader(mask, f"{r.where}.mask").integer("size", None) if mask is not None else None
        dim = r.integer("dim")
        return cls(heads=heads, kv_heads=kv, dim=dim, vdim=r.integer("vdim", dim),
                   scale=r.number("scale", positive=False), window=window,
                   rot=Rotation.read(r.data.get("rot"), f"{r.where}.rot", dim), v_mix=r.boolean("v_mix", False))

    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale, "v_mix": self.v_mix}
        if self.window is not None:
            d["mask"] = {"size": self.window}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    def part(self, hidden: int, eps: float) -> PartSpec:
        return PartSpec("sink_rotary_attention", {
            "hidden_size": hidden, "heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim,
            "vdim": self.vdim, "rot_dims": self.rot.dims if self.rot else 0, "scale": self.scale,
            "window": self.window, "eps": eps, "unit_norm": False, "sink": False, "bias": False,
            "value_mix": self.mix_role})


@dataclass(frozen=True)
class LatentAttentionLayer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[Rotation]

    type = "latent_attention"

    @classmethod
    def read(cls, r: KeyReader) -> "LatentAttentionLayer":
        rot_dim = r.integer("rot_dim", 0, minimum=0)
        dim = r.integer("dim")
        rot = Rotation.read(r.data.get("rot"), f"{r.where}.rot", rot_dim, exactly=True) if rot_dim else None
        return cls(heads=r.integer("heads"), dim=dim, rot_dim=rot_dim, vdim=r.integer("vdim", dim),
                   kv_rank=r.integer("kv_rank"), scale=r.number("scale", positive=False), rot=rot)

    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim,
                             "kv_rank": self.kv_rank, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    def part(self, hidden: int, eps: float) -> PartSpec:
        return PartSpec("latent_attention", {
            "hidden_size": hidden, "heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim,
            "vdim": self.vdim, "q_rank": None, "kv_rank": self.kv_rank, "window": None, "scale": self.scale,
            "eps": eps, "rot_dims": self.rot.dims if self.rot else 0, "gate": "head", "sink": False})


@dataclass(frozen=True)
class SelectiveScanLayer:
    inner: int
    state: int
    dt_rank: int
    conv: int

    type = "mamba1"
    rot = None

    @classmethod
    def read(cls, r: KeyReader) -> "SelectiveScanLayer":
        return cls(inner=r.integer("inner"), state=r.integer("state"), dt_rank=r.integer("dt_rank"),
                   conv=r.integer("conv"))

    def to_dict(self) -> dict:
        return {"inner": self.inner, "state": self.state, "dt_rank": self.dt_rank, "conv": self.conv}

    def part(self, hidden: int, eps: float) -> PartSpec:
        return PartSpec("mamba1", {"hidden_size": hidden, **self.to_dict()})


@dataclass(frozen=True)
class DenseFeedForward:
    ff: int

    kind = "dense"

    @classmethod
    def read(cls, r: KeyReader) -> "DenseFeedForward":
        return cls(ff=r.integer("ff"))

    def to_dict(self) -> dict:
        return {"kind": self.kind, "ff": self.ff}

    def part(self, hidden: int) -> PartSpec:
        return PartSpec("swiglu", {"hidden_size": hidden, "intermediate_size": self.ff,
                                   "tensor_names": SWIGLU_NAMES})


MIXERS = {c.type: c for c in (WindowAttentionLayer, LatentAttentionLayer, SelectiveScanLayer)}
FEED_FORWARDS = {c.kind: c for c in (DenseFeedForward,)}


@dataclass(frozen=True)
class BeralixLayer:
    mixer: Any                     # one of the classes in MIXERS
    mlp: Any                       # one of the classes in FEED_FORWARDS, or None: the layer has none


def _with_mix_roles(layers, where: str):
    """The layers with mixed values told apart: the first one gives its values, the later ones take them."""
    first, out = None, []
    for i, l in enumerate(layers):
        m = l.mixer
        if getattr(m, "v_mix", False):
            if first is None:
                first = m
            elif (m.kv_heads, m.vdim) != (first.kv_heads, first.vdim):
                raise ConfigError(f"{where}: layers[{i}].mixer: its {m.kv_heads} value heads of {m.vdim} cannot be mixed "
                                  f"with the first such layer's {first.kv_heads} of {first.vdim}")
            l = BeralixLayer(replace(m, mix_role="first" if m is first else "later"), l.mlp)
        out.append(l)
    return tuple(out)


@dataclass(frozen=True)
class BeralixConfig:
    width: int
    vocab: int
    layers: Tuple[BeralixLayer, ...]
    eps: float
    logit_softcap: Optional[float]
    max_position_embeddings: int = 4096         # the default size of the cache, no bound of the design
    architecture: str = "Beralix"

    @classmethod
    def from_dict(cls, data: dict, where: str = "config.json") -> "BeralixConfig":
        r = KeyReader(data, where)
        norm = KeyReader(data.get("norm"), f"{where}: norm")
        layers = []
        for i, entry in enumerate(r.list_of("layers")):
            lr = KeyReader(entry, f"{where}: layers[{i}]")
            kind = lr.string("type")
            if kind not in MIXERS:
                raise ConfigError(f"{where}: layers[{i}].type '{kind}' is not known; known: {', '.join(sorted(MIXERS))}")
            mixer = MIXERS[kind].read(KeyReader(entry.get("mixer"), f"{where}: layers[{i}].mixer"))
            mlp, ff = entry.get("mlp"), None
            if mlp is not None:
                mr = KeyReader(mlp, f"{where}: layers[{i}].mlp")
                ff_kind = mr.string("kind", "dense")
                if ff_kind not in FEED_FORWARDS:
                    raise ConfigError(f"{where}: layers[{i}].mlp.kind '{ff_kind}' is not known; known: "
                                      f"{', '.join(sorted(FEED_FORWARDS))}")
                ff = FEED_FORWARDS[ff_kind].read(mr)
            layers.append(BeralixLayer(mixer, ff))
        if not layers:
            raise ConfigError(f"{where}: 'layers' is empty")
        return cls(width=r.integer("width"), vocab=r.integer("vocab"), layers=_with_mix_roles(layers, where),
                   eps=norm.number("eps"), logit_softcap=r.number("logit_softcap", None),
                   max_position_embeddings=r.integer("max_position_embeddings", 4096),
                   architecture=r.string("architecture", "Beralix"))

    def to_dict(self) -> dict:
        """The config.json dictionary that reads back to this configuration."""
        d: Dict[str, Any] = {
            "architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
            "layers": [{"type": l.mixer.type, "mixer": l.mixer.to_dict(),
                        "mlp": None if l.mlp is None else l.mlp.to_dict()} for l in self.layers]}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("layernorm", {"size": self.width, "eps": self.eps})
        layers = []
        for i, l in enumerate(self.layers):
            prefix, rot = f"l{i}", l.mixer.rot
            params = {"prefix": prefix, "size": self.width}
            if l.mlp is None:
                block, ff = PartSpec("sandwich_mixer_only", {**params, "scales": (MIXER_SCALE,)}), PartSpec("none")
                norms = {"mixer_norm": norm, "mixer_out_norm": norm}
                # without a feed-forward its norms and factor are not used; a folder that stores them all the
                # same is accepted
                second = (LAYER_TENSOR_NAMES["feed_forward_norm"], LAYER_TENSOR_NAMES["feed_forward_out_norm"])
                unused = {n: (self.width,) for s in second for n in (s, s + ".b")}
                unused[FEED_FORWARD_SCALE] = (self.width,)
            else:
                block = PartSpec("sandwich", {**params, "scales": (MIXER_SCALE, FEED_FORWARD_SCALE)})
                ff = l.mlp.part(self.width)
                norms = {"mixer_norm": norm, "mixer_out_norm": norm, "feed_forward_norm": norm,
                         "feed_forward_out_norm": norm}
                unused = {}
            layers.append(LayerSpec(prefix=prefix, block=block, mixer=l.mixer.part(self.width, self.eps),
                                    feed_forward=ff, norms=norms, names=LAYER_TENSOR_NAMES,
                                    position=rot.part() if rot else None, unused_tensors=unused))
        spec = ModelSpec(hidden_size=self.width, vocab_size=self.vocab, embedding_name="embed", head_name="head",
                         tie_head_to_embedding=False, final_norm=norm, final_norm_prefix="final.norm",
                         layers=tuple(layers), order=tuple(range(len(layers))), stop_token_ids=(),
                         logit_softcap=self.logit_softcap)
        spec.validate()
        return spec

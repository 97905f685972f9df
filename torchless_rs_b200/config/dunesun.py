"""Typed configuration of the Dunesun decoder, read from its config.json.

The design: the stream starts as the token's row plus a learned row of its position.  A layer is a parallel
block, x <- x + (mixer(N(x)) + ff(N(x))), N an RMS norm whose stored weight lies around zero; the mixer is one of
  * `attention`: softmax attention with grouped key/value heads, queries and keys RMS-normed over the whole
    projection, no rotation, a sliding window (`mask.size`), and one added to the softmax's denominator;
  * `mamba2`: a state-space recurrence with one decay per head and token behind a short causal convolution of
    `conv` taps, gated and then normed in `norm_groups` equal parts.
The feed-forward is a mixture of SwiGLU experts weighed by a softmax over the chosen experts' logits, with an
optional shared expert behind a sigmoid gate (`mlp.shared`), or absent (`mlp` null).  `loop` lets the layers
start .. stop - 1 run `times` times in a row with the same weights and a cache per pass; before each pass a row
of the table `loop.step` is added to the stream, and before each pass but the first the embedded token again.
The logits are multiplied by `logit_scale`.  config.json lists the layers one by one with all their sizes and
constants (`layers[i].type`, `.mixer`, `.mlp`), so layers of one model may differ in all of them.  Tensor names:
`embed`, `pos`, `loop.step`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .errors import ConfigError
from .reader import KeyReader
from .spec import LayerSpec, ModelSpec, PartSpec, PassStart

LAYER_TENSOR_NAMES = {"norm": "norm1", "mixer": "mix", "feed_forward": "mlp"}
SINK_LOGIT = 0.0          # the sink that adds one to the softmax's denominator: fixed by the design


@dataclass(frozen=True)
class WindowAttentionLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]

    type = "attention"

    @classmethod
    def read(cls, r: KeyReader) -> "WindowAttentionLayer":
        heads, kv = r.integer("heads"), r.integer("kv_heads")
        if heads % kv:
            raise ConfigError(f"{r.where}: 'heads' {heads} is no multiple of 'kv_heads' {kv}")
        mask = r.data.get("mask")
        window = KeyReader(mask, f"{r.where}.mask").integer("size") if mask is not None else None
        dim = r.integer("dim")
        return cls(heads=heads, kv_heads=kv, dim=dim, vdim=r.integer("vdim", dim),
                   scale=r.number("scale", positive=False), window=window)

    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale}
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d

    def part(self, hidden: int, eps: float) -> PartSpec:
        return PartSpec("sink_window_attention", {
            "hidden_size": hidden, "heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
            "window": self.window, "keep_first": 0, "scale": self.scale, "softcap": None, "eps": eps, "bias": False,
            "gate": False, "sink": SINK_LOGIT, "qk_norm": "whole"})


@dataclass(frozen=True)
class StateSpaceLayer:
    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int

    type = "mamba2"

    @classmethod
    def read(cls, r: KeyReader) -> "StateSpaceLayer":
        heads, groups, vdim = r.integer("heads"), r.integer("groups", 1), r.integer("vdim")
        parts = r.integer("norm_groups", 1)
        if heads % groups:
            raise ConfigError(f"{r.where}: 'heads' {heads} is no multiple of 'groups' {groups}")
        if heads * vdim % parts:
            raise ConfigError(f"{r.where}: {heads} heads of {vdim} have no {parts} equal parts ('norm_groups')")
        return cls(heads=heads, groups=groups, state=r.integer("state"), vdim=vdim, conv=r.integer("conv"),
                   norm_groups=parts)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "groups": self.groups, "state": self.state, "vdim": self.vdim, "conv": self.conv,
                "norm_groups": self.norm_groups}

    def part(self, hidden: int, eps: float) -> PartSpec:
        return PartSpec("mamba2", {"hidden_size": hidden, "eps": eps, **self.to_dict()})


@dataclass(frozen=True)
class ExpertFeedForward:
    ff: int
    experts: int
    top: int
    shared_ff: Optional[int]

    kind = "moe"

    @classmethod
    def read(cls, r: KeyReader) -> "ExpertFeedForward":
        for key in ("expert", "router"):
            if not isinstance(r.data.get(key), dict):
                raise ConfigError(f"{r.where}: required key '{key}' is missing")
        router = KeyReader(r.data["router"], f"{r.where}.router")
        experts, top = router.integer("experts"), router.integer("top")
        if top > experts:
            raise ConfigError(f"{router.where}: 'top' {top} is more than the {experts} experts there are")
        shared = r.data.get("shared")
        return cls(ff=KeyReader(r.data["expert"], f"{r.where}.expert").integer("ff"), experts=experts, top=top,
                   shared_ff=KeyReader(shared, f"{r.where}.shared").integer("ff") if shared is not None else None)

    def to_dict(self) -> dict:
        d: Dict[str, Any] = {"kind": self.kind, "expert": {"ff": self.ff},
                             "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff is not None:
            d["shared"] = {"ff": self.shared_ff}
        return d

    def part(self, hidden: int) -> PartSpec:
        return PartSpec("moe_softmax_chosen", {"hidden_size": hidden, "ff": self.ff, "experts": self.experts,
                                               "top": self.top, "shared_ff": self.shared_ff})


MIXERS = {c.type: c for c in (WindowAttentionLayer, StateSpaceLayer)}
FEED_FORWARDS = {c.kind: c for c in (ExpertFeedForward,)}


@dataclass(frozen=True)
class DunesunLayer:
    mixer: Any                     # one of the classes in MIXERS
    mlp: Any                       # one of the classes in FEED_FORWARDS, or None: the layer has none


@dataclass(frozen=True)
class Loop:
    """Layers start .. stop - 1 run `times` times in a row."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class DunesunConfig:
    width: int
    vocab: int
    layers: Tuple[DunesunLayer, ...]
    loop: Optional[Loop]
    eps: float
    logit_scale: float
    max_positions: int
    architecture: str = "Dunesun"

    @property
    def max_position_embeddings(self) -> int:
        """The default size of the cache: a sequence cannot be longer than the position table."""
        return self.max_positions

    @classmethod
    def from_dict(cls, data: dict, where: str = "config.json") -> "DunesunConfig":
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
                ff_kind = mr.string("kind", "moe")
                if ff_kind not in FEED_FORWARDS:
                    raise ConfigError(f"{where}: layers[{i}].mlp.kind '{ff_kind}' is not known; known: "
                                      f"{', '.join(sorted(FEED_FORWARDS))}")
                ff = FEED_FORWARDS[ff_kind].read(mr)
            layers.append(DunesunLayer(mixer, ff))
        if not layers:
            raise ConfigError(f"{where}: 'layers' is empty")
        loop = None
        if data.get("loop") is not None:
            pr = KeyReader(data["loop"], f"{where}: loop")
            loop = Loop(start=pr.integer("start", minimum=0), stop=pr.integer("stop"), times=pr.integer("times"))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"{where}: loop: 'start' {loop.start} and 'stop' {loop.stop} name no layers of the "
                                  f"{len(layers)} there are")
        return cls(width=r.integer("width"), vocab=r.integer("vocab"), layers=tuple(layers), loop=loop,
                   eps=norm.number("eps"), logit_scale=r.number("logit_scale", 1.0, positive=False),
                   max_positions=r.integer("max_positions"), architecture=r.string("architecture", "Dunesun"))

    def to_dict(self) -> dict:
        """The config.json dictionary that reads back to this configuration."""
        d: Dict[str, Any] = {
            "architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
            "logit_scale": self.logit_scale, "max_positions": self.max_positions,
            "layers": [{"type": l.mixer.type, "mixer": l.mixer.to_dict(),
                        "mlp": None if l.mlp is None else l.mlp.to_dict()} for l in self.layers]}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return d

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("rmsnorm_one_plus", {"size": self.width, "eps": self.eps})
        final = PartSpec("rmsnorm_one_plus", {"size": self.width, "eps": self.eps, "output_scale": self.logit_scale})
        layers = [LayerSpec(prefix=f"l{i}", block=PartSpec("parallel_sublayers"), mixer=l.mixer.part(self.width, self.eps),
                            feed_forward=PartSpec("none") if l.mlp is None else l.mlp.part(self.width),
                            norms={"norm": norm}, names=LAYER_TENSOR_NAMES) for i, l in enumerate(self.layers)]
        order, starts = list(range(len(layers))), {}
        if self.loop is not None:
            p = self.loop
            run = list(range(p.start, p.stop))
            order = list(range(p.start)) + run * p.times + list(range(p.stop, len(layers)))
            starts = {p.start + t * len(run): PassStart(row=t, add_embedded=t > 0) for t in range(p.times)}
        spec = ModelSpec(hidden_size=self.width, vocab_size=self.vocab, embedding_name="embed", head_name="head",
                         tie_head_to_embedding=False, final_norm=final, final_norm_prefix="final.norm",
                         layers=tuple(layers), order=tuple(order), stop_token_ids=(), position_table_name="pos",
                         max_positions=self.max_positions, pass_starts=starts,
                         pass_table_name="loop.step" if self.loop is not None else None,
                         pass_rows=self.loop.times if self.loop is not None else 0)
        spec.validate()
        return spec

"""The arrangement of parts in a layer.  Pre-norm residual block:
h += mixer(norm1(h)); h += feed_forward(norm2(h)); the residual is the stream before
the norm (reference: src/model/modules/layer.rs:28-56).  The stream stays in 32-bit
and each part adds into it."""
from __future__ import annotations

import torch

from ..weights.loader import TensorSpec
from .registry import register_block
from .runtime import Runtime


@register_block("prenorm")
class PreNormBlock:
    """Interface of every block: a class attribute `norm_roles` (the norms this kind of block
    takes; a layer's spec must give exactly these), a constructor `(spec, rt, mixer,
    feed_forward, norms)` with `norms` a dictionary by role, the attributes `mixer`,
    `feed_forward` and `norms`, and `forward(x, batch)`, which updates the 32-bit stream `x`
    [tokens, hidden] in place.

    Optional, for blocks that let the products around a norm take it over: `takes_carry =
    True`, `first_norm` (the norm whose input the block before may prepare; None if its mixer
    cannot use one) and `forward(x, batch, carry, next_norm)` returning a carry for
    `next_norm` or None.  A block without `takes_carry` is called with `(x, batch)` only."""
    norm_roles = ("mixer_norm", "feed_forward_norm")
    takes_carry = True

    def __init__(self, spec, rt: Runtime, mixer, feed_forward, norms):
        self.rt = rt
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = dict(norms)
        self.mixer_norm = norms["mixer_norm"]
        self.feed_forward_norm = norms["feed_forward_norm"]

    @property
    def first_norm(self):
        return self.mixer_norm if getattr(self.mixer, "accepts_carry", False) else None

    def forward(self, x: torch.Tensor, batch, carry=None, next_norm=None):
        """`carry`: the input of this block's first norm if the product before it prepared
        it (else None).  `next_norm`: the norm that follows this block; the block returns
        a carry for it if its last product could prepare one (else None).

        A norm is folded into its neighbours only if it says it is `foldable` and both
        neighbours say they `accepts_carry`; otherwise the norm kernel runs."""
        from .linear import new_carry
        rt = self.rt
        xn = rt.workspace.get("block_normed", x.shape, rt.act_dtype)
        fold = not rt.is_f32

        def can_fold(norm, producer, consumer):
            return (fold and norm is not None and getattr(norm, "foldable", False)
                    and getattr(producer, "accepts_carry", False)
                    and getattr(consumer, "accepts_carry", False))

        inp = carry if (carry is not None and carry.valid) else self.mixer_norm(x, xn)
        c2 = None
        if can_fold(self.feed_forward_norm, self.mixer, self.feed_forward):
            c2 = new_carry(rt, "a", x.shape[0], self.feed_forward_norm.size, self.feed_forward_norm.eps)
            self.mixer.forward(inp, x, batch, emit=(self.feed_forward_norm.weight, c2))
        else:
            self.mixer.forward(inp, x, batch)
        inp2 = c2 if (c2 is not None and c2.valid) else self.feed_forward_norm(x, xn)
        c3 = None
        if next_norm is not None and getattr(next_norm, "foldable", False) and fold and \
                getattr(self.feed_forward, "accepts_carry", False):
            c3 = new_carry(rt, "b", x.shape[0], next_norm.size, next_norm.eps)
            self.feed_forward.forward(inp2, x, batch, emit=(next_norm.weight, c3))
        else:
            self.feed_forward.forward(inp2, x, batch)
        return c3 if (c3 is not None and c3.valid) else None


@register_block("prenorm_mixer_only")
class PreNormMixerBlock:
    """The pre-norm block of a layer without a feed-forward: x += mixer(norm1(x))."""
    norm_roles = ("mixer_norm",)

    def __init__(self, spec, rt: Runtime, mixer, feed_forward, norms):
        self.rt = rt
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = dict(norms)
        self.mixer_norm = norms["mixer_norm"]

    def forward(self, x: torch.Tensor, batch) -> None:
        rt = self.rt
        xn = rt.workspace.get("block_normed", x.shape, rt.act_dtype)
        self.mixer.forward(self.mixer_norm(x, xn), x, batch)


class StreamCopy:
    """What a branch-norm block hands to the next one: the stream in the activation type, as the
    kernel that last changed the stream wrote it.  (`valid` is False so that a block that expects the
    prepared input of a norm ignores it.)"""
    valid = False

    def __init__(self, xb: torch.Tensor):
        self.xb = xb


@register_block("branchnorm")
class BranchNormBlock:
    """x <- x + m * norm_1(mixer(x)); x <- x + m * norm_2(feed_forward(x)): the sublayers read the
    stream itself and the norm sits on each branch's output.  Parameter: `residual_mult` (m).

    The branch writes its output to a 32-bit buffer; one kernel takes its root mean square, adds
    m * gain * y / rms to the stream and writes the stream's copy in the activation type, which the next
    sublayer's products read (in 32-bit the stream is that copy).  A sublayer that says
    `can_overwrite` stores its output (`forward(..., overwrite=True)`); any other adds into the zeroed
    buffer, so every registered mixer and feed-forward fits.  Norms: any with a single `gain`, or
    with a `weight` per coordinate."""
    norm_roles = ("mixer_out_norm", "feed_forward_out_norm")
    takes_carry = True
    first_norm = None   # no norm stands before this block's first product

    def __init__(self, spec, rt: Runtime, mixer, feed_forward, norms):
        self.rt = rt
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = dict(norms)
        self.mult = float(spec.get("residual_mult", 1.0))
        self._gains = {}

    def _gain(self, norm):
        g = getattr(norm, "gain", None)
        if g is not None:
            return g
        key = id(norm)
        if key not in self._gains:
            self._gains[key] = norm.weight.to(torch.float32).contiguous()
        return self._gains[key]

    def _branch(self, part, norm, x, xb, batch):
        rt = self.rt
        y = rt.workspace.get("branch_out", x.shape, torch.float32)
        if getattr(part, "can_overwrite", False):
            part.forward(xb, y, batch, overwrite=True)
        else:
            y.zero_()
            part.forward(xb, y, batch)
        gain = self._gain(norm)
        if gain.numel() != 1:
            # a weight per coordinate: the norm's own kernel, then the scaled sum
            yn = rt.workspace.get("branch_normed", x.shape, rt.act_dtype)
            norm(y, yn)
            x.add_(yn.to(torch.float32), alpha=self.mult)
            if xb is not x:
                xb.copy_(x)
            return
        rt.ops.branch_norm_add(y, gain, self.mult, norm.eps, x, None if xb is x else xb)

    def forward(self, x: torch.Tensor, batch, carry=None, next_norm=None):
        rt = self.rt
        if rt.is_f32:
            xb = x
        elif isinstance(carry, StreamCopy) and carry.xb.shape == x.shape:
            xb = carry.xb
        else:
            xb = rt.workspace.get("branch_in", x.shape, rt.act_dtype)
            rt.ops.convert_into(x, xb)
        self._branch(self.mixer, self.norms["mixer_out_norm"], x, xb, batch)
        if "feed_forward_out_norm" in self.norms:
            self._branch(self.feed_forward, self.norms["feed_forward_out_norm"], x, xb, batch)
        return None if xb is x else StreamCopy(xb)


@register_block("branchnorm_mixer_only")
class BranchNormMixerBlock(BranchNormBlock):
    """The same block for a layer without a feed-forward: x <- x + m * norm_1(mixer(x))."""
    norm_roles = ("mixer_out_norm",)


class NormedInput:
    """What a sandwich block hands to the next one: the next block's first norm already applied to the
    stream, written by the kernel that last changed the stream.  (`valid` is False so that a block that
    expects the prepared input of a folded norm ignores it.)"""
    valid = False

    def __init__(self, xn: torch.Tensor, norm):
        self.xn, self.norm = xn, norm


@register_block("sandwich")
class SandwichBlock:
    """x <- x + N_1b(mixer(N_1(x))); x <- x + N_2b(feed_forward(N_2(x))): a norm before and after every
    sublayer, each with its own weight.

    A sublayer writes its output to a 32-bit buffer (one that says `can_overwrite` stores it, any other adds
    into the zeroed buffer, so every registered mixer and feed-forward fits); one kernel norms that output,
    adds it to the stream and applies the norm that comes next (this block's second, or the next block's
    first, which is handed on as a `NormedInput`), so the stream crosses memory once per sublayer.  The
    fused kernel takes norms with a plain weight per coordinate (`weight`, `eps`), and layer norms (`bias`
    too); the next norm is fused only if it is of the same kind and its weight has the same type as this one's.

    Optional parameters: `scales`, the names under `prefix` of one vector per sublayer (of `size` numbers) that
    multiplies what the sublayer's output norm gives.  They are taken into that norm's weight and bias when the
    weights come in (32-bit)."""
    norm_roles = ("mixer_norm", "mixer_out_norm", "feed_forward_norm", "feed_forward_out_norm")
    takes_carry = True

    def __init__(self, spec, rt: Runtime, mixer, feed_forward, norms):
        self.rt = rt
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = dict(norms)
        self.scales = tuple(spec.get("scales") or ())
        self.prefix = str(spec.get("prefix") or "")
        self._scaled = {}        # output norm's role -> (weight, bias) with the sublayer's scale in them

    @classmethod
    def expected_tensors(cls, spec, prefix: str):
        return {f"{prefix}.{n}": TensorSpec((int(spec.params["size"]),)) for n in (spec.get("scales") or ())}

    def load(self, weights) -> None:
        for role, name in zip(("mixer_out_norm", "feed_forward_out_norm"), self.scales):
            norm = self.norms[role]
            s = weights[f"{self.prefix}.{name}"].to(device=self.rt.device, dtype=torch.float32)
            bias = getattr(norm, "bias", None)
            self._scaled[role] = ((norm.weight.to(torch.float32) * s).contiguous(),
                                  (bias * s).contiguous() if bias is not None else None)

    @property
    def first_norm(self):
        return self.norms["mixer_norm"]

    def _sublayer(self, part, role, x, xn, batch, next_norm):
        """x += norms[role](part(xn)); returns next_norm(x) if it could be taken along, else None."""
        rt, norm_out = self.rt, self.norms[role]
        weight, bias = self._scaled.get(role) or (norm_out.weight, getattr(norm_out, "bias", None))
        y = rt.workspace.get("branch_out", x.shape, torch.float32)
        if getattr(part, "can_overwrite", False):
            part.forward(xn, y, batch, overwrite=True)
        else:
            y.zero_()
            part.forward(xn, y, batch)
        fuse = (next_norm is not None and getattr(next_norm, "weight", None) is not None
                and getattr(next_norm, "size", None) == x.shape[1]
                and next_norm.weight.dtype == weight.dtype
                and (getattr(next_norm, "bias", None) is None) == (bias is None))
        out = rt.workspace.get("block_normed", x.shape, rt.act_dtype) if fuse else None
        if bias is not None:
            then = (next_norm.weight, next_norm.bias, next_norm.eps, out) if fuse else ()
            rt.ops.layernorm_add_layernorm(y, weight, bias, norm_out.eps, x, *then)
        else:
            rt.ops.norm_add_norm(y, weight, norm_out.eps, x, *((next_norm.weight, next_norm.eps, out) if fuse else ()))
        return out

    def _input(self, norm, x, carry):
        if isinstance(carry, NormedInput) and carry.norm is norm and carry.xn.shape == x.shape:
            return carry.xn
        return norm(x, self.rt.workspace.get("block_normed", x.shape, self.rt.act_dtype))

    def forward(self, x: torch.Tensor, batch, carry=None, next_norm=None):
        n = self.norms
        xn = self._input(n["mixer_norm"], x, carry)
        second = n.get("feed_forward_norm")
        got = self._sublayer(self.mixer, "mixer_out_norm", x, xn, batch, second if second is not None else next_norm)
        if second is None:
            return NormedInput(got, next_norm) if got is not None else None
        xn = got if got is not None else second(x, self.rt.workspace.get("block_normed", x.shape, self.rt.act_dtype))
        got = self._sublayer(self.feed_forward, "feed_forward_out_norm", x, xn, batch, next_norm)
        return NormedInput(got, next_norm) if got is not None else None


@register_block("sandwich_mixer_only")
class SandwichMixerBlock(SandwichBlock):
    """The same block for a layer without a feed-forward: x <- x + N_1b(mixer(N_1(x)))."""
    norm_roles = ("mixer_norm", "mixer_out_norm")


@register_block("parallel_sublayers")
class ParallelSublayersBlock:
    """x <- x + (mixer(h) + feed_forward(h)), h = N(x): one norm, both sublayers read its output.  Takes layers
    with and without a feed-forward (part "none").

    The mixer's output projection adds into the stream.  A feed-forward that offers `terms` leaves its last sum
    to the block's closing kernel, which also takes what comes between this layer and the next (`addend`) and
    the next norm, so the stream crosses memory once for all of them; any other feed-forward adds into the
    stream itself.  Where the mixer can hold rows for the feed-forward in its input product (`take_rows`) and
    the feed-forward names some (`input_rows`), both share that product.  The closing kernel takes next norms
    with a 32-bit weight per coordinate (`weight`, `eps`)."""
    norm_roles = ("norm",)
    takes_carry = True
    takes_addend = True

    def __init__(self, spec, rt: Runtime, mixer, feed_forward, norms):
        self.rt = rt
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = dict(norms)
        self.shares_input = hasattr(mixer, "take_rows") and hasattr(feed_forward, "input_rows")
        if self.shares_input:
            mixer.take_rows(feed_forward.input_rows())
            feed_forward.own_input = False

    @property
    def first_norm(self):
        return self.norms["norm"]

    def forward(self, x: torch.Tensor, batch, carry=None, next_norm=None, addend=None):
        """`addend` = (rows [tokens, hidden] or None, vector [hidden] or None): added to the stream after the
        layer, before `next_norm`."""
        rt, norm = self.rt, self.norms["norm"]
        if isinstance(carry, NormedInput) and carry.norm is norm and carry.xn.shape == x.shape:
            xn = carry.xn
        else:
            xn = norm(x, rt.workspace.get("block_normed", x.shape, rt.act_dtype))
        self.mixer.forward(xn, x, batch)
        experts = shared = None
        if hasattr(self.feed_forward, "terms"):
            experts, shared = self.feed_forward.terms(xn, batch, self.mixer.row_products if self.shares_input else None)
        else:
            self.feed_forward.forward(xn, x, batch)
        w = getattr(next_norm, "weight", None)
        fuse = w is not None and w.dtype == torch.float32 and w.numel() == x.shape[1]
        if not fuse and experts is None and shared is None and addend is None:
            return None
        rows, vec = addend if addend is not None else (None, None)
        if not fuse:
            rt.ops.close_block(x, experts, shared, rows, vec)
            return None
        out = rt.workspace.get("block_normed", x.shape, rt.act_dtype)
        rt.ops.close_block(x, experts, shared, rows, vec, w, next_norm.eps, out)
        return NormedInput(out, next_norm)

"""A selective state-space recurrence with one decay per head and token (Mamba-2): a matrix state per head that
decays by a number computed from the token and is written with the token's own step size.

With h the mixer's input, per token (`heads` heads of `vdim`, `groups` groups of `state` entries; head n reads
group n // (heads / groups)):
    [z | x | B | C | dt] = W_in h
    [x | B | C] <- silu(conv([x | B | C]) + b)      conv: over the last `conv` tokens of each channel, zeros
                                                    before the sequence's start
    dt <- softplus(dt + dt_bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T,   y = S^T C + D x                       (per head)
    out = W_o ( N(y silu(z)) )      N: RMS norm of each of `norm_groups` equal parts of the row, one weight
S starts at zero, is 32-bit and is carried from token to token in the cache's per-sequence state together
with the convolution's last `conv` - 1 inputs (two `StateRequest`s), so a prompt may come in any number of
pieces.  Step sizes, decays, state, gate and norm are 32-bit; x, B and C are of the activation type."""
from __future__ import annotations

from typing import Dict

import torch

from ..cache.requests import StateRequest
from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorSpec
from .linear import InputRows, Matmul
from .registry import register_mixer
from .runtime import Runtime


@register_mixer("mamba2")
class StateSpaceDuality(InputRows):
    """Parameters: `hidden_size`, `heads`, `groups`, `state`, `vdim`, `conv` (taps), `norm_groups`, `eps` (of the
    output norm).  Tensors under the prefix: in, conv, conv.b, dt_bias, A_log, D, norm, o."""
    graph_safe = True
    can_overwrite = True
    state_attributes = ("state", "kept", "row_products")

    def __init__(self, spec: PartSpec, prefix: str, rt: Runtime, position=None):
        p = spec.params
        self.heads, self.groups = int(p["heads"]), int(p["groups"])
        self.n, self.vdim, self.taps = int(p["state"]), int(p["vdim"]), int(p["conv"])
        self.parts = int(p.get("norm_groups") or 1)
        self.eps = float(p["eps"])
        if self.heads % self.groups:
            raise ValueError(f"{self.heads} heads cannot share {self.groups} groups")
        if self.taps < 1:
            raise ValueError("a convolution needs at least one tap")
        self.inner = self.heads * self.vdim
        if self.inner % self.parts:
            raise ValueError(f"a row of {self.inner} has no {self.parts} equal parts")
        self.channels = self.inner + 2 * self.groups * self.n
        self.prefix = prefix
        self.rt = rt
        self.matmul = Matmul(rt)
        self.state = None
        self.kept = None

    @classmethod
    def expected_tensors(cls, spec: PartSpec, prefix: str) -> Dict[str, TensorSpec]:
        p = spec.params
        hidden, H, G, N, P, taps = (int(p[k]) for k in ("hidden_size", "heads", "groups", "state", "vdim", "conv"))
        inner = H * P
        channels = inner + 2 * G * N
        return {
            f"{prefix}.in": TensorSpec((inner + channels + H, hidden), init=(hidden ** -0.5, 0.0)),
            f"{prefix}.conv": TensorSpec((channels, taps), init=(0.5, 0.0)),
            f"{prefix}.conv.b": TensorSpec((channels,), init=(0.1, 0.0)),
            f"{prefix}.dt_bias": TensorSpec((H,), init=(1.0, -2.0)),
            f"{prefix}.A_log": TensorSpec((H,), init=(0.7, 0.5)),
            f"{prefix}.D": TensorSpec((H,), init=(0.3, 1.0)),
            f"{prefix}.norm": TensorSpec((inner,)),
            f"{prefix}.o": TensorSpec((hidden, inner), init=(inner ** -0.5, 0.0)),
        }

    def load(self, weights: Dict[str, torch.Tensor]) -> None:
        p, rt = self.prefix, self.rt
        self.w_in = self.stack_input(rt, weights, [weights[f"{p}.in"]])
        self.w_o = rt.matrix(weights[f"{p}.o"])
        f32 = lambda t: t.to(device=rt.device, dtype=torch.float32).contiguous()
        self.taps_w = f32(weights[f"{p}.conv"])
        self.conv_b = f32(weights[f"{p}.conv.b"])
        self.dt_bias = f32(weights[f"{p}.dt_bias"])
        self.neg_a = -torch.exp(f32(weights[f"{p}.A_log"]))       # the decay's rate, 32-bit, once
        self.D = f32(weights[f"{p}.D"])
        self.norm_w = f32(weights[f"{p}.norm"])

    def cache_request(self):
        return (StateRequest((self.heads, self.n, self.vdim), torch.float32),
                StateRequest((max(self.taps - 1, 1), self.channels), torch.float32))

    def bind_cache(self, views) -> None:
        self.state, self.kept = views       # [slots, heads, state, vdim], [slots, taps - 1, channels]

    def forward(self, xn: torch.Tensor, residual: torch.Tensor, batch, emit=None, overwrite: bool = False) -> None:
        rt, ws = self.rt, self.rt.workspace
        T = residual.shape[0]
        z = self.project_input(xn, "ssd_in", T)
        xbc = ws.get("ssd_xbc", (T, self.channels), rt.act_dtype)
        dtla = ws.get("ssd_steps", (T, self.heads, 2), torch.float32)
        rt.ops.ssd_prep(z, self.inner, self.inner + self.channels, self.taps_w, self.conv_b, self.kept, xbc, dtla,
                        self.neg_a, self.dt_bias, batch.seq_start, batch.seq_slot)
        y = ws.get("ssd_out", (T, self.inner), torch.float32)
        rt.ops.ssd_scan(xbc, dtla, self.D, self.state, y, batch.seq_start, batch.seq_slot, self.heads, self.groups,
                        workspace=ws)
        gated = ws.get("ssd_gated", (T, self.inner), rt.act_dtype)
        rt.ops.ssd_gate_norm(y, z[:, :self.inner], self.norm_w, self.eps, gated, self.parts)
        self.matmul(gated, self.w_o, residual, ops.MODE_STORE_F32 if overwrite else ops.MODE_ACCUM_F32)

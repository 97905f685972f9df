"""A selective scan (Mamba): a state of `state` numbers per channel, each of which decays by a number of its own
that the token's step size sets, behind a short causal convolution.

With h the mixer's input, per token (`inner` channels):
    [x | z] = W_in h
    x <- silu(conv(x) + b)                conv: over the last `conv` tokens of each channel, zeros before the
                                          sequence's start
    [d | B | C] = W_x x                   d of `dt_rank` numbers, B and C of `state`
    dt = softplus(W_dt d + b_dt)          one step size per channel
    S_c,n <- exp(dt_c A_c,n) S_c,n + dt_c x_c B_n,   y_c = sum_n S_c,n C_n + D_c x_c       A = -exp(A_log)
    out = W_o (y silu(z))
S starts at zero, is 32-bit and is carried from token to token in the cache's per-sequence state together
with the convolution's last `conv` - 1 inputs (two `StateRequest`s), so a prompt may come in any number of
pieces.  Step sizes, decays, state and gate are 32-bit; x, z, d, B and C are of the activation type.

The columns of d are padded to a multiple of 8 with zero rows of W_x and zero columns of W_dt, so that the
second product reads its rows on 16-byte boundaries."""
from __future__ import annotations

from typing import Dict

import torch

from ..cache.requests import StateRequest
from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorSpec
from .linear import Matmul
from .registry import register_mixer
from .runtime import Runtime


@register_mixer("mamba1")
class SelectiveScan:
    """Parameters: `hidden_size`, `inner` (channels), `state` (entries per channel), `dt_rank`, `conv` (taps).
    Tensors under the prefix: in, conv, conv.b, x, dt, dt.b, A_log, D, o."""
    graph_safe = True
    can_overwrite = True
    state_attributes = ("state", "kept")

    def __init__(self, spec: PartSpec, prefix: str, rt: Runtime, position=None):
        p = spec.params
        self.inner, self.n = int(p["inner"]), int(p["state"])
        self.rank, self.taps = int(p["dt_rank"]), int(p["conv"])
        if position is not None:
            raise ValueError("a selective scan takes no positional rotation")
        self.rank_pad = -(-self.rank // 8) * 8
        self.prefix = prefix
        self.rt = rt
        self.matmul = Matmul(rt)
        self.state = None
        self.kept = None

    @classmethod
    def expected_tensors(cls, spec: PartSpec, prefix: str) -> Dict[str, TensorSpec]:
        p = spec.params
        hidden, inner, N, R, taps = (int(p[k]) for k in ("hidden_size", "inner", "state", "dt_rank", "conv"))
        return {
            f"{prefix}.in": TensorSpec((2 * inner, hidden), init=(hidden ** -0.5, 0.0)),
            f"{prefix}.conv": TensorSpec((inner, taps), init=(0.5, 0.0)),
            f"{prefix}.conv.b": TensorSpec((inner,), init=(0.1, 0.0)),
            f"{prefix}.x": TensorSpec((R + 2 * N, inner), init=(inner ** -0.5, 0.0)),
            f"{prefix}.dt": TensorSpec((inner, R), init=(R ** -0.5, 0.0)),
            f"{prefix}.dt.b": TensorSpec((inner,), init=(1.0, -2.0)),
            f"{prefix}.A_log": TensorSpec((inner, N), init=(0.7, 0.5)),
            f"{prefix}.D": TensorSpec((inner,), init=(0.3, 1.0)),
            f"{prefix}.o": TensorSpec((hidden, inner), init=(inner ** -0.5, 0.0)),
        }

    def load(self, weights: Dict[str, torch.Tensor]) -> None:
        p, rt = self.prefix, self.rt
        R, pad = self.rank, self.rank_pad - self.rank
        w_x, w_dt = weights[f"{p}.x"], weights[f"{p}.dt"]
        rows = [w_x[:R].contiguous(), torch.zeros((pad, self.inner), dtype=w_x.dtype, device=w_x.device),
                w_x[R:].contiguous(),
                torch.zeros((-(self.rank_pad + 2 * self.n) % 8, self.inner), dtype=w_x.dtype, device=w_x.device)]
        self.w_in = rt.matrix(weights[f"{p}.in"])
        self.w_x = rt.stack([r for r in rows if r.shape[0]])
        self.w_dt = rt.matrix(torch.nn.functional.pad(w_dt, (0, pad)) if pad else w_dt)
        self.w_o = rt.matrix(weights[f"{p}.o"])
        f32 = lambda t: t.to(device=rt.device, dtype=torch.float32).contiguous()
        self.taps_w = f32(weights[f"{p}.conv"])
        self.conv_b = f32(weights[f"{p}.conv.b"])
        self.dt_bias = f32(weights[f"{p}.dt.b"])
        self.neg_a = -torch.exp(f32(weights[f"{p}.A_log"]))       # the decays' rates, 32-bit, once
        self.D = f32(weights[f"{p}.D"])

    def cache_request(self):
        return (StateRequest((self.inner, self.n), torch.float32),
                StateRequest((max(self.taps - 1, 1), self.inner), torch.float32))

    def bind_cache(self, views) -> None:
        self.state, self.kept = views       # [slots, inner, state], [slots, taps - 1, inner]

    def forward(self, xn: torch.Tensor, residual: torch.Tensor, batch, emit=None, overwrite: bool = False) -> None:
        rt, ws = self.rt, self.rt.workspace
        T, inner = residual.shape[0], self.inner
        xz = ws.get("scan1_in", (T, 2 * inner), rt.act_dtype)
        self.matmul(xn, self.w_in, xz, ops.MODE_STORE_ACT)
        x = ws.get("scan1_x", (T, inner), rt.act_dtype)
        rt.ops.conv_silu(xz, 0, self.taps_w, self.conv_b, self.kept, x, batch.seq_start, batch.seq_slot)
        dbc = ws.get("scan1_dbc", (T, self.w_x.shape[0]), rt.act_dtype)
        self.matmul(x, self.w_x, dbc, ops.MODE_STORE_ACT)
        dt = ws.get("scan1_dt", (T, inner), torch.float32)
        self.matmul(dbc[:, :self.rank_pad], self.w_dt, dt, ops.MODE_STORE_F32)
        y = ws.get("scan1_y", (T, inner), rt.act_dtype)
        rt.ops.selective_scan(x, dt, self.dt_bias, dbc, self.rank_pad, self.neg_a, self.D, xz[:, inner:], self.state, y,
                              batch.seq_start, batch.seq_slot)
        self.matmul(y, self.w_o, residual, ops.MODE_STORE_F32 if overwrite else ops.MODE_ACCUM_F32)

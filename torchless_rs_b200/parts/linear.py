"""Matrix products of the parts: picks the kernel for a shape.

`out (op)= a @ w.T` with 32-bit accumulation.  In 32-bit everything runs on the
CUDA-core kernels.  In bfloat16 the tensor-core kernels take the shapes they are
built for and the CUDA-core kernels take the rest; which kernel ran never changes
what is computed, only its rounding order.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .runtime import Runtime


class NormCarry:
    """The input of a norm that the product before it has already prepared: `xw` = the
    stream times the norm's weight (bfloat16), `ss` = partial sums of squares of each row
    of the stream, one per 128 columns.  The product after it scales its outputs by
    1/rms.  `valid` says whether the last producer filled it."""

    def __init__(self, xw: torch.Tensor, ss: torch.Tensor, size: int, eps: float):
        self.xw, self.ss, self.size, self.eps = xw, ss, size, eps
        self.tiles = ss.shape[1]
        self.valid = False


def new_carry(rt: Runtime, name: str, n_tokens: int, size: int, eps: float) -> NormCarry:
    ws = rt.workspace
    tiles = (size + 127) // 128
    return NormCarry(ws.get(f"carry_xw_{name}", (n_tokens, size), torch.bfloat16),
                     ws.get(f"carry_ss_{name}", (n_tokens, tiles), torch.float32), size, eps)


class Matmul:
    def __init__(self, rt: Runtime):
        self.rt = rt
        self.fast = None
        if not rt.is_f32:
            from ..csrc import gemm_bf16
            self.fast = gemm_bf16.GemmBf16.get()

    def __call__(self, a, w: torch.Tensor, out: torch.Tensor, mode: int, emit=None, rope=None) -> bool:
        """`a` is an activation tensor or a `NormCarry`.  `emit` = (norm weight, NormCarry)
        asks the product (mode 1) to prepare the next norm's input if it can.  `rope` (a
        `gemm_bf16.RopeArgs`) asks the q/k/v product to rotate and write q, k and v itself;
        the return value says whether it did (then `out` was not written)."""
        scaled = a if isinstance(a, NormCarry) else None
        if scaled is not None:
            if self.fast is None or not self.fast.run(scaled.xw, w, out, mode, scaled=scaled, rope=rope):
                raise ops.KernelError("a folded norm reached a product that cannot apply it")
            return self.fast.rope_applied
        if emit is not None:
            emit[1].valid = False
        if self.fast is not None and self.fast.run(a, w, out, mode, emit=emit, rope=rope):
            return self.fast.rope_applied
        self.rt.ops.gemm_generic(a, w, out, mode)
        return False

    def activated(self, a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, mode: int, act) -> bool:
        """The product with another activation in its epilogue than the mode's own (`act` as
        `GemmBf16.run` takes it): True if the tensor-core kernel took it, False if the caller has to
        run the product into 32-bit and the activation as a kernel of its own."""
        return self.fast is not None and self.fast.run(a, w, out, mode, act=act)


class InputRows:
    """For a mixer whose input goes through one stacked product into 32-bit: lets the feed-forward beside it,
    which reads the same input, have rows of its own in that product (a router's, a gate's).

    `take_rows(names)` (before `load`) names matrices to be stacked below the mixer's own;
    `stack_input` makes the stacked matrix, `project_input` runs the product, and `row_products` is then the
    [tokens, rows] view of what the taken rows gave, valid until the next product of this kind."""
    row_names: tuple = ()
    row_products = None

    def take_rows(self, names) -> None:
        self.row_names = tuple(names)

    def stack_input(self, rt: Runtime, weights, own) -> torch.Tensor:
        mats = list(own) + [weights[n] for n in self.row_names]
        self.own_rows = sum(int(m.shape[0]) for m in own)
        self.taken_rows = sum(int(weights[n].shape[0]) for n in self.row_names)
        pad = -(self.own_rows + self.taken_rows) % 8       # rows of 32-bit results start on 16-byte boundaries
        if pad:
            mats.append(torch.zeros((pad, mats[0].shape[1]), dtype=mats[0].dtype, device=mats[0].device))
        return rt.stack(mats)

    def project_input(self, xn: torch.Tensor, name: str, T: int) -> torch.Tensor:
        z = self.rt.workspace.get(name, (T, self.w_in.shape[0]), torch.float32)
        self.matmul(xn, self.w_in, z, ops.MODE_STORE_F32)
        if self.taken_rows:
            self.row_products = z[:, self.own_rows:self.own_rows + self.taken_rows]
        return z

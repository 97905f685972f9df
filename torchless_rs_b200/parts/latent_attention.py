"""Attention whose keys and values are reconstructed from a low-rank latent, with a rotated key
part shared by all heads; optionally a sliding window, a sigmoid output gate (per entry or per head) and
a sink logit per head in the softmax's denominator.

With h the mixer's input, per token:
    c_q = norm(W_dq h) * w_q,        q = W_uq c_q        (per head: `dim` plain + `rot_dim` rotated),
                                     or, without a query latent, q = W_q h
    [c' | r'] = W_dkv h,             c = norm(c') * w_c,  r = rotate(r')
    k_h = [W_uk,h c | r],  v_h = W_uv,h c,  score = (q_h . k_h) * scale over the window
    p(i, j) = exp(score(i, j)) / (sum over visible j' of exp(score(i, j')) [+ exp(sink_h)])
    out = W_o ((heads' weighted values, concatenated) [* sigmoid(W_g h)])
Only [c | r] is cached, one vector per position (`PagedLatentRequest`).  Keys and values are
never formed: q's plain part is carried into the latent space (W_uk,h^T q_h), the weighted sum
is taken over the c's, and W_uv,h is applied to the sum, so prefill and decode run the same
kernels on the same pages and a position's result does not depend on the step that computes it.
The projections of h (W_dq or W_q, W_dkv and, with a gate, W_g) are one stacked product.

The rotated parts of a query and of the shared key only ever meet in their dot product, which does
not change when both are permuted alike.  A model whose rotation pairs entries (2i, 2i + 1) (the
position part's style) is therefore run by the kernels for pairs (i, i + n/2): the rows of
W_uq's rotated part and of W_dkv's last rows are reordered once, when the weights come in."""
from __future__ import annotations

import math
from typing import Dict

import torch

from ..cache.requests import PagedLatentRequest
from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorSpec
from .linear import Matmul
from .registry import register_mixer
from .runtime import Runtime


@register_mixer("latent_attention")
class LatentAttention:
    """Parameters: `hidden_size`, `heads`, `dim` (plain query/key size per head), `rot_dim` (rotated
    size), `vdim`, `q_rank` (None: queries straight from the input), `kv_rank`, `window` (None = all keys), `scale` (default
    1/sqrt(dim + rot_dim)), `eps` (of the two latent norms), `rot_dims` (how many of the rot_dim
    entries turn; default all), `gate` (True or "entry", the default: a sigmoid gate per output entry, tensor g
    [heads * vdim, hidden]; "head": one per head, g [heads, hidden]; False: none), `sink`
    (default False: a learned logit per head, tensor sink).  The position part gives the frequencies of
    `rot_dims` entries and the pairing.
    Tensors under the prefix: dq, dq.norm, uq (without a query latent: q), dkv, dkv.norm, uk, uv, [g], [sink], o."""
    graph_safe = True
    can_overwrite = True
    FEW_TOKENS = 16     # up to here a step keeps W_uq and W_uk apart

    def __init__(self, spec: PartSpec, prefix: str, rt: Runtime, position=None):
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.heads = int(p["heads"])
        self.dim = int(p["dim"])
        self.rot = int(p["rot_dim"])
        self.vdim = int(p["vdim"])
        self.q_rank = int(p.get("q_rank") or 0)
        self.rank = int(p["kv_rank"])
        self.window = int(p["window"]) if p.get("window") else None
        self.eps = float(p["eps"])
        self.rot_dims = int(p.get("rot_dims", self.rot)) if position is not None else 0
        self.gate_rows = self._gate_rows(p)
        self.has_sink = bool(p.get("sink", False))
        # the layer's position part names the pairing, as for the other rotated mixers
        self.pairing = "interleaved" if getattr(position, "style", 0) == 1 else "half_split"
        self.amplitude = float(getattr(position, "amplitude", 1.0))
        self.sink = None
        self.scale = float(p["scale"]) if p.get("scale") else 1.0 / math.sqrt(self.dim + self.rot)
        if self.rot_dims > self.rot or self.rot_dims % 2:
            raise ValueError(f"{self.rot_dims} rotated entries do not fit a rotated part of {self.rot}")
        if position is not None and self.rot_dims and position.inv_freq.numel() != self.rot_dims // 2:
            raise ValueError("the position part's frequencies do not fit the rotated entries")
        self.prefix = prefix
        self.rt = rt
        self.position = position
        self.matmul = Matmul(rt)
        self.cache = None

    @staticmethod
    def _shapes(p):
        H, dim, rot, vdim = int(p["heads"]), int(p["dim"]), int(p["rot_dim"]), int(p["vdim"])
        return int(p["hidden_size"]), H, dim, rot, vdim, int(p.get("q_rank") or 0), int(p["kv_rank"])

    @staticmethod
    def _gate_rows(p) -> int:
        """Rows of the gate's matrix: one per output entry, one per head, or none."""
        kind = p.get("gate", True)
        if kind not in (True, False, "entry", "head"):
            raise ValueError(f"a gate is per 'entry', per 'head' or absent, not '{kind}'")
        return 0 if kind is False else int(p["heads"]) * (1 if kind == "head" else int(p["vdim"]))

    @classmethod
    def expected_tensors(cls, spec: PartSpec, prefix: str) -> Dict[str, TensorSpec]:
        hidden, H, dim, rot, vdim, q_rank, rank = cls._shapes(spec.params)
        queries = {
            f"{prefix}.dq": TensorSpec((q_rank, hidden)),
            f"{prefix}.dq.norm": TensorSpec((q_rank,)),
            f"{prefix}.uq": TensorSpec((H * (dim + rot), q_rank)),
        } if q_rank else {f"{prefix}.q": TensorSpec((H * (dim + rot), hidden))}
        out = {
            **queries,
            f"{prefix}.dkv": TensorSpec((rank + rot, hidden)),
            f"{prefix}.dkv.norm": TensorSpec((rank,)),
            f"{prefix}.uk": TensorSpec((H * dim, rank)),
            f"{prefix}.uv": TensorSpec((H * vdim, rank)),
            f"{prefix}.o": TensorSpec((hidden, H * vdim)),
        }
        if cls._gate_rows(spec.params):
            out[f"{prefix}.g"] = TensorSpec((cls._gate_rows(spec.params), hidden))
        if spec.params.get("sink", False):
            out[f"{prefix}.sink"] = TensorSpec((H,), init=(1.0, 0.0))
        return out

    def _reordered(self, t: torch.Tensor, first: int) -> torch.Tensor:
        """Rows first .. first + rot_dims of `t` so that the pair (2i, 2i + 1) becomes (i, i + rot_dims/2)."""
        n = self.rot_dims
        if self.pairing != "interleaved" or n == 0:
            return t
        order = list(range(0, n, 2)) + list(range(1, n, 2))
        t = t.clone()
        t[first:first + n] = t[first:first + n][order]
        return t

    def load(self, weights: Dict[str, torch.Tensor]) -> None:
        p, rt = self.prefix, self.rt
        w_dkv = self._reordered(weights[f"{p}.dkv"], self.rank)
        w_q = weights[f"{p}.uq" if self.q_rank else f"{p}.q"]
        w_q = w_q.reshape(self.heads, self.dim + self.rot, w_q.shape[-1])
        w_q = torch.stack([self._reordered(w_q[h], self.dim) for h in range(self.heads)]) \
            .reshape(self.heads * (self.dim + self.rot), w_q.shape[-1])
        gate = [weights[f"{p}.g"]] if self.gate_rows else []
        if self.q_rank:
            self.w_in = rt.stack([weights[f"{p}.dq"], w_dkv] + gate)
            self.w_uq = rt.matrix(w_q)
        else:
            rows = w_q.shape[0] + w_dkv.shape[0] + self.gate_rows
            pad = torch.zeros((-rows % 8, w_q.shape[1]), dtype=w_q.dtype, device=w_q.device)
            self.w_in = rt.stack([w_q, w_dkv] + gate + ([pad] if pad.shape[0] else []))   # 16-byte rows of results
        # per head, transposed: the query's plain part is multiplied by W_uk,h^T
        uk = weights[f"{p}.uk"].reshape(self.heads, self.dim, self.rank).transpose(1, 2).contiguous()
        self.w_uk_t = rt.matrix(uk)                                          # [heads, rank, dim]
        self.w_uv = rt.matrix(weights[f"{p}.uv"].reshape(self.heads, self.vdim, self.rank))
        self.w_o = rt.matrix(weights[f"{p}.o"])
        f32 = lambda t: t.to(device=rt.device, dtype=torch.float32).contiguous()
        self.norm_q = f32(weights[f"{p}.dq.norm"]) if self.q_rank else None
        self.norm_c = f32(weights[f"{p}.dkv.norm"])
        if self.has_sink:
            self.sink = f32(weights[f"{p}.sink"])
        if not self.q_rank:
            return
        # For steps of many tokens W_uk,h^T is folded into W_uq: one product gives every head's
        # [latent-space query | part to rotate].  (Folded in 64-bit, once, when the weights come in.)
        uq64 = w_q.to(device=rt.device, dtype=torch.float64).reshape(
            self.heads, self.dim + self.rot, self.q_rank)
        uk64 = weights[f"{p}.uk"].to(device=rt.device, dtype=torch.float64).reshape(self.heads, self.dim, self.rank)
        folded = torch.cat([torch.bmm(uk64.transpose(1, 2), uq64[:, :self.dim]), uq64[:, self.dim:]], dim=1)
        self.w_q_latent = rt.matrix(folded.reshape(self.heads * (self.rank + self.rot), self.q_rank)
                                    .to(torch.float32 if rt.is_f32 else torch.bfloat16))
        del uq64, uk64, folded

    def cache_request(self):
        return PagedLatentRequest(self.rank + self.rot, self.window)

    def bind_cache(self, view) -> None:
        self.cache = view

    def forward(self, xn: torch.Tensor, residual: torch.Tensor, batch, emit=None, overwrite: bool = False) -> None:
        rt, ws, o = self.rt, self.rt.workspace, self.rt.ops
        T = residual.shape[0]
        H, dim, rot, rank, vdim, q_rank = self.heads, self.dim, self.rot, self.rank, self.vdim, self.q_rank
        c = self.cache
        inv_freq = self.position.inv_freq if self.rot_dims else None
        n_q = q_rank or H * (dim + rot)          # columns of the input product ahead of the latent's
        g_off = n_q + rank + rot
        s = ws.get("latent_in", (T, self.w_in.shape[0]), torch.float32)
        self.matmul(xn, self.w_in, s, ops.MODE_STORE_F32)
        dkv = s[:, n_q:g_off]
        cq = ws.get("latent_cq", (T, q_rank), rt.act_dtype) if q_rank else None
        o.latent_prep(s[:, :q_rank] if q_rank else None, dkv, self.norm_q, self.norm_c, self.eps, cq, c.pages,
                      batch.token_pos, batch.token_seq, batch.seq_slot, c.page_table, inv_freq, rank, rot,
                      self.rot_dims, amplitude=self.amplitude)
        mix = ws.get("latent_mix", (T, H, rank), torch.float32)
        if not q_rank or T <= self.FEW_TOKENS:
            # without a query latent, or for few tokens (two small matrices are fewer bytes to stream than the
            # folded one): the queries, then their plain parts into the latent space
            q = s
            if q_rank:
                q = ws.get("latent_q", (T, H * (dim + rot)), torch.float32)
                self.matmul(cq, self.w_uq, q, ops.MODE_STORE_F32)
            qa, qa_head, q_off = ws.get("latent_qa", (T, H * rank), torch.float32), rank, dim
            o.headwise_gemm(q, dim + rot, self.w_uk_t, qa, rank)
            q_head = dim + rot
        else:
            q = ws.get("latent_ql", (T, H * (rank + rot)), torch.float32)
            self.matmul(cq, self.w_q_latent, q, ops.MODE_STORE_F32)
            qa, qa_head, q_head, q_off = q, rank + rot, rank + rot, rank
        o.latent_attn(qa, qa_head, q, q_head, q_off, c.pages, mix, batch.token_pos, batch.token_seq, batch.seq_slot,
                      c.page_table, inv_freq, H, rank, rot, self.rot_dims, self.window, self.scale,
                      max_keys=batch.len_bucket, workspace=ws, sink=self.sink, amplitude=self.amplitude)
        gated = ws.get("latent_gated", (T, H * vdim), rt.act_dtype)
        o.headwise_gemm(mix.view(T, H * rank), rank, self.w_uv, gated, vdim,
                        gate=s[:, g_off:g_off + self.gate_rows] if self.gate_rows else None, act_out=True)
        self.matmul(gated, self.w_o, residual, ops.MODE_STORE_F32 if overwrite else ops.MODE_ACCUM_F32)

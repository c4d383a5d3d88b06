"""A linear attention whose memory fades per key channel (gated linear attention), as a mixer with per-sequence state.

    q = Wq x1 * dim^-1/2,  k = Wk x1  (heads x dim),   v = Wv x1,  gate = silu(Wg x1)  (heads x vdim)
    alpha = sigmoid(A2 (A1 x1) + bias)^(1 / tau)          per head and key channel
    per head:  S <- diag(alpha) S + k v^T;   o = S^T q    (the token itself included)
    out = Wo (o / rms_head(o) * norm * gate)

S is zero when a sequence starts, float, and carried from step to step in the engine's per-sequence state (one row per
slot).  Decays, their logarithms and exponentials, the state and the per-head norm are float on both paths; A1's product
writes float and enters the second one without loss (its error would add up along the sequence); the bfloat16 path
differs in the type of q, k, v and the gate.  Kernels: csrc/gated_linear.cu and, for prompts, the scan of
csrc/decay_memory.cu.
"""
from __future__ import annotations

import torch

from ..csrc import lib
from .base import MIXERS, Mixer, ParamDecl, StateNeed
from .linear import matmul_nt

USE_STEP = True         # one token per sequence: the kernel that does everything between the projections and the output


def split_width(rank: int, dtype: torch.dtype) -> int:
    """Entries of a row that enters a decay's second product: in bfloat16 two halves, the value and what its rounding
    left."""
    return rank if dtype == torch.float32 else 2 * ((rank + 3) // 4 * 4)


def split_weight(w: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """The second product's weight for such rows: what the rounding left is a second half of the row, so the matrix
    stands there twice."""
    if dtype == torch.float32:
        return w
    half = torch.cat([w, w.new_zeros((w.shape[0], split_width(w.shape[1], dtype) // 2 - w.shape[1]))], dim=1)
    return torch.cat([half, half], dim=1).contiguous()


@MIXERS.register("gated_linear")
class GatedLinear(Mixer):
    """params: width, heads, dim, vdim, tau, rank, eps; optional: out_scale (default 1)."""
    graph_safe = True
    launches_only = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        g = lambda n: int(params[n])
        self.d, self.H, self.dim, self.vdim, self.rank = g("width"), g("heads"), g("dim"), g("vdim"), g("rank")
        self.tau, self.eps = float(params["tau"]), float(params["eps"])
        self.out_scale = float(params.get("out_scale", 1.0))
        if min(self.H, self.dim, self.vdim, self.rank) <= 0 or not self.tau > 0:
            raise ValueError("heads, dim, vdim, rank and tau must be positive")
        if self.dim > 256:
            raise ValueError(f"the gated linear attention's kernels take heads of up to 256 key entries, got {self.dim}")
        self.hk, self.hv = self.H * self.dim, self.H * self.vdim
        self.rows_width = self.hv
        self.in_weight, self.in_width = "win", 2 * self.hk + 2 * self.hv

    def parameters(self):
        return {
            "win": ParamDecl((self.in_width, self.d)),             # rows: q heads, k heads, v heads, output gate
            "a1": ParamDecl((self.rank, self.d)),
            "a2": ParamDecl((self.hk, self.rank)),
            "a2_bias": ParamDecl((self.hk,), "norm", "normal"),
            "norm": ParamDecl((self.vdim,), "norm", "ones"),
            "wo": ParamDecl((self.d, self.hv)),
        }

    def bind(self, tensors) -> None:
        super().bind(tensors)
        self.weights["a2_split"] = split_weight(self.weights["a2"], self.dtype)
        # the kernels that norm the heads' outputs take one weight per (head, entry): the shared one, repeated
        self.weights["norm"] = (self.weights["norm"].float() * self.out_scale).repeat(self.H).contiguous()

    def state_need(self):
        return StateNeed(((self.hk * self.vdim + 3) // 4 * 4,), torch.float32)

    def forward_rows(self, ctx, x1, rows, cache, state, z=None) -> None:
        nt, H = x1.shape[0], self.H
        sfx = lib.suffix(self.dtype)
        w = self.weights
        pitch = state.stride(0)
        if z is None:
            z = ctx.scratch("gla.z", (nt, self.in_width), self.dtype)
            matmul_nt(x1, w["win"], z)
        ldz = z.stride(0)
        a = ctx.scratch("gla.a", (nt, self.rank), torch.float32)
        matmul_nt(x1, w["a1"], a)                                           # float out on both paths
        if ctx.decode and USE_STEP and lib.try_call(
                "tb_gated_linear_step_" + sfx, lib.ptr(z), ldz, lib.ptr(a), self.rank, lib.ptr(w["a2"]),
                lib.ptr(w["a2_bias"]), lib.ptr(w["norm"]), lib.ptr(state), pitch, lib.ptr(rows), rows.stride(0),
                lib.ptr(ctx.seq_start), lib.ptr(ctx.slots), nt, ctx.B, H, self.dim, self.vdim, self.rank, 1.0 / self.tau,
                self.dim ** -0.5, self.eps):
            return
        split = ctx.scratch("gla.split", (nt, split_width(self.rank, self.dtype)), self.dtype)
        lib.call("tb_split_rows_" + sfx, lib.ptr(a), self.rank, lib.ptr(split), nt, self.rank, split.shape[1])
        pre = ctx.scratch("gla.pre", (nt, self.hk), torch.float32)
        matmul_nt(split, w["a2_split"], pre)                                # float out
        size = lib.gated_linear_record_size(self.dim, self.vdim)
        rec = ctx.scratch("gla.rec", (H, nt, size), torch.float32)
        lib.call("tb_gated_linear_prep_" + sfx, lib.ptr(z), ldz, lib.ptr(pre), lib.ptr(w["a2_bias"]), lib.ptr(rec),
                 nt, H, self.dim, self.vdim, size, 1.0 / self.tau, self.dim ** -0.5)
        o = ctx.scratch("gla.o", (nt, self.hv), torch.float32)
        lib.call("tb_decay_scan_rect", lib.ptr(rec), lib.ptr(state), pitch, lib.ptr(o), lib.ptr(ctx.seq_start),
                 lib.ptr(ctx.slots), nt, ctx.B, H, self.dim, self.vdim)
        gate = z[:, 2 * self.hk + self.hv:]
        lib.call("tb_mlstm_out_" + sfx, lib.ptr(o), lib.ptr(gate), ldz, lib.ptr(w["norm"]), lib.ptr(rows), nt, H,
                 self.vdim, self.eps, 1, rows.stride(0))

    def forward(self, ctx, x1, out, cache, state, z=None) -> None:
        rows = ctx.scratch("gla.y", (x1.shape[0], self.hv), self.dtype)
        self.forward_rows(ctx, x1, rows, cache, state, z)
        matmul_nt(rows, self.weights["wo"], out)

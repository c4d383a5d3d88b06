"""A delta rule in which the decay, the removal and the key that is written are made separately (the time mixing of the
RWKV-7 family), as a mixer with per-sequence state.

    r, k, v = Wr x1, Wk x1, Wv x1,   gate = sigmoid(Wg x1)                        (heads x dim)
    w = exp(-e^(-1/2) sigmoid(W2 tanh(W1 x1) + w0)),   a = sigmoid(Wa x1 + ba)    per head and key channel
    per head, u = k / sqrt(sum k^2 + 1e-6):
        S <- diag(w) S - (a u)(u^T S) + k v^T   (both terms read the old S);   o = S^T r
    out = Wo (o / rms_head(o) * norm * gate * out_scale)

S is zero when a sequence starts, float, and carried from step to step in the engine's per-sequence state (one row per
slot).  Decays, removal rates, unit keys, the state and the per-head norm are float on both paths; the projections of the
removal rate and of the decay share a product that writes float (their error would add up along the sequence); the
bfloat16 path differs in the type of r, k, v and the gate.  Kernels: csrc/split_delta.cu.
"""
from __future__ import annotations

import torch

from ..csrc import lib
from .base import MIXERS, Mixer, ParamDecl, StateNeed
from .gated_linear import split_weight, split_width
from .linear import matmul_nt

USE_STEP = True         # one token per sequence: the kernel that does everything between the projections and the output


@MIXERS.register("split_delta")
class SplitDelta(Mixer):
    """params: width, heads, dim, rank, eps; optional: out_scale (default 1)."""
    graph_safe = True
    launches_only = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        g = lambda n: int(params[n])
        self.d, self.H, self.dim, self.rank = g("width"), g("heads"), g("dim"), g("rank")
        self.eps = float(params["eps"])
        self.out_scale = float(params.get("out_scale", 1.0))
        if min(self.H, self.dim, self.rank) <= 0:
            raise ValueError("heads, dim and rank must be positive")
        if self.dim > 256:
            raise ValueError(f"the split delta rule's kernels take heads of up to 256 entries, got {self.dim}")
        self.rows_width = self.hd = self.H * self.dim
        self.in_weight, self.in_width = "win", 4 * self.hd

    def parameters(self):
        return {
            "win": ParamDecl((4 * self.hd, self.d)),              # rows: r heads, k heads, v heads, output gate
            "wa": ParamDecl((self.hd + self.rank, self.d)),       # rows: removal rate, the decay's first projection
            "ba": ParamDecl((self.hd,), "norm", "normal"),
            "w2": ParamDecl((self.hd, self.rank)),
            "w0": ParamDecl((self.hd,), "norm", "normal"),
            "norm": ParamDecl((self.hd,), "norm", "ones"),
            "wo": ParamDecl((self.d, self.hd)),
        }

    def bind(self, tensors) -> None:
        super().bind(tensors)
        self.weights["w2_split"] = split_weight(self.weights["w2"], self.dtype)
        if self.out_scale != 1.0:
            self.weights["norm"] = (self.weights["norm"].float() * self.out_scale).contiguous()

    def state_need(self):
        return StateNeed(((self.hd * self.dim + 3) // 4 * 4,), torch.float32)

    def forward_rows(self, ctx, x1, rows, cache, state, z=None) -> None:
        nt, H, hd = x1.shape[0], self.H, self.hd
        sfx = lib.suffix(self.dtype)
        w = self.weights
        pitch = state.stride(0)
        if z is None:
            z = ctx.scratch("sdelta.z", (nt, 4 * hd), self.dtype)
            matmul_nt(x1, w["win"], z)
        ldz = z.stride(0)
        wide = hd + self.rank
        az = ctx.scratch("sdelta.a", (nt, wide), torch.float32)
        matmul_nt(x1, w["wa"], az)                                          # float out on both paths
        if ctx.decode and USE_STEP and lib.try_call(
                "tb_split_delta_step_" + sfx, lib.ptr(z), ldz, lib.ptr(az), wide, lib.ptr(w["ba"]), lib.ptr(w["w2"]),
                lib.ptr(w["w0"]), lib.ptr(w["norm"]), self.eps, lib.ptr(state), pitch, lib.ptr(rows), rows.stride(0),
                lib.ptr(ctx.seq_start), lib.ptr(ctx.slots), nt, ctx.B, H, self.dim, self.rank):
            return
        th = ctx.scratch("sdelta.tanh", (nt, split_width(self.rank, self.dtype)), self.dtype)
        lib.call("tb_decay_tanh_" + sfx, lib.ptr(az[:, hd:]), wide, lib.ptr(th), nt, self.rank, th.shape[1])
        pre = ctx.scratch("sdelta.pre", (nt, hd), torch.float32)
        matmul_nt(th, w["w2_split"], pre)                                   # float out
        rec = ctx.scratch("sdelta.rec", (H, nt, lib.split_delta_record_size(self.dim)), torch.float32)
        lib.call("tb_split_delta_prep_" + sfx, lib.ptr(z), ldz, lib.ptr(az), wide, lib.ptr(w["ba"]), lib.ptr(pre),
                 lib.ptr(w["w0"]), lib.ptr(rec), nt, H, self.dim)
        o = ctx.scratch("sdelta.o", (nt, hd), torch.float32)
        lib.call("tb_split_delta_scan", lib.ptr(rec), lib.ptr(state), pitch, lib.ptr(o), lib.ptr(ctx.seq_start),
                 lib.ptr(ctx.slots), nt, ctx.B, H, self.dim)
        lib.call("tb_mlstm_out_" + sfx, lib.ptr(o), lib.ptr(z[:, 3 * hd:]), ldz, lib.ptr(w["norm"]), lib.ptr(rows), nt, H,
                 self.dim, self.eps, 0, rows.stride(0))

    def forward(self, ctx, x1, out, cache, state, z=None) -> None:
        rows = ctx.scratch("sdelta.y", (x1.shape[0], self.hd), self.dtype)
        self.forward_rows(ctx, x1, rows, cache, state, z)
        matmul_nt(rows, self.weights["wo"], out)

"""A linear memory with a decay per key channel made from the input, a bonus for the current token and a shift of the
input by one token (the time mixing of the RWKV family), as a mixer with per-sequence state.

    mix_m[t] = x1[t] + (x1[t-1] - x1[t]) mu_m        m in r, k, v, g, w;   x1[-1] = 0 when a sequence starts
    r, k, v = Wr mix_r, Wk mix_k, Wv mix_v  (heads x dim)        gate = silu(Wg mix_g)
    w = exp(-exp(w0 + W2 tanh(W1 mix_w)))                        per head and key channel
    per head:  o = S^T r + (r . (u k)) v;    S <- diag(w) S + k v^T
    out = Wo (o / rms_head(o) * norm * gate * out_scale)

S and the last input are state of the sequence, float, one row per slot.  Decays with both exponentials, the small
product W2 tanh(.), the bonus, the state and the per-head norm are float on both paths; W1's product writes float (its
error would add up along the sequence); the bfloat16 path differs in the type of the mixes and of r, k, v and the gate.
Kernels: csrc/decay_memory.cu: all mixes in one, the four wide projections as ONE grouped product (a matrix per mix);
then for prompts decays and records, the scan, norm and gate; for one token per sequence all of that in one kernel.
"""
from __future__ import annotations

import torch

from ..csrc import lib
from . import linear
from .base import MIXERS, Mixer, ParamDecl, StateNeed
from .linear import gemm_skinny, grouped_matmul, matmul_nt

USE_STEP = True         # one token per sequence: the kernel that does everything between the projections and the output

GROUPS = 4              # r, k, v, gate: mixes with a wide matrix each


@MIXERS.register("decay_memory")
class DecayMemory(Mixer):
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
            raise ValueError(f"the decaying memory's kernels take heads of up to 256 entries, got {self.dim}")
        if self.rank > 1024:
            raise ValueError(f"the decaying memory's kernels take ranks up to 1024, got {self.rank}")
        self.rows_width = self.hd = self.H * self.dim
        # a row of tanh values for the product with W2: in bfloat16 two halves (the value, what its rounding left)
        self.tanh_width = self.rank if dtype == torch.float32 else 2 * ((self.rank + 3) // 4 * 4)

    def parameters(self):
        return {
            "mu": ParamDecl((GROUPS + 1, self.d), "norm", "normal"),          # r, k, v, gate, decay
            "win": ParamDecl((GROUPS, self.hd, self.d)),                      # r, k, v, gate
            "w1": ParamDecl((self.rank, self.d)),
            "w2": ParamDecl((self.hd, self.rank)),
            "w0": ParamDecl((self.hd,), "norm", "normal"),
            "u": ParamDecl((self.H, self.dim), "norm", "normal"),
            "norm": ParamDecl((self.hd,), "norm", "ones"),
            "wo": ParamDecl((self.d, self.hd)),
        }

    def bind(self, tensors) -> None:
        super().bind(tensors)
        w2 = self.weights["w2"]
        if self.dtype == torch.float32:
            self.weights["w2_tanh"] = w2
        else:       # what tanh's rounding leaves is a second half of the product's rows: W2 stands there again
            half = torch.cat([w2, w2.new_zeros((self.hd, self.tanh_width // 2 - self.rank))], dim=1)
            self.weights["w2_tanh"] = torch.cat([half, half], dim=1).contiguous()
        if self.out_scale != 1.0:
            self.weights["norm"] = (self.weights["norm"].float() * self.out_scale).contiguous()

    def state_need(self):
        return StateNeed((lib.decay_state_size(self.H, self.dim, self.d),), torch.float32)

    def forward_rows(self, ctx, x1, rows, cache, state) -> None:
        nt, d, H, hd = x1.shape[0], self.d, self.H, self.hd
        sfx = lib.suffix(self.dtype)
        w = self.weights
        pitch = state.stride(0)
        mixes = ctx.scratch("decay.mixes", ((GROUPS + 1) * nt, d), self.dtype)
        offsets = ctx.scratch("decay.offsets", (GROUPS + 1,), torch.int32)
        few = self.dtype == torch.bfloat16 and GROUPS * nt <= linear.SKINNY_MAX_PAIRS
        group = ctx.scratch("decay.group", (GROUPS * nt,), torch.int32) if few else None
        lib.call("tb_shift_mix_" + sfx, lib.ptr(x1), lib.ptr(w["mu"]), lib.ptr(state), pitch, H * self.dim * self.dim,
                 lib.ptr(mixes), lib.ptr(offsets), lib.ptr(group), GROUPS, lib.ptr(ctx.tok_seq), lib.ptr(ctx.seq_start),
                 lib.ptr(ctx.slots), nt, d)
        wide = mixes[:GROUPS * nt]
        z = ctx.scratch("decay.z", (GROUPS * nt, hd), self.dtype)           # r, k, v, gate: nt rows each
        if not (few and gemm_skinny(wide, w["win"], z, groups=GROUPS, max_group_rows=nt, row_group=group)):
            grouped_matmul(wide, w["win"], z, group_offsets=offsets, groups=GROUPS, max_group_rows=nt)
        a = ctx.scratch("decay.a", (nt, self.rank), torch.float32)
        matmul_nt(mixes[GROUPS * nt:], w["w1"], a)                          # float out on both paths
        if ctx.decode and USE_STEP and lib.try_call(
                "tb_decay_step_" + sfx, lib.ptr(z), lib.ptr(x1), d, lib.ptr(a), self.rank, lib.ptr(w["w2"]),
                lib.ptr(w["w0"]), lib.ptr(w["u"]), lib.ptr(w["norm"]), self.eps, lib.ptr(state), pitch, lib.ptr(rows),
                rows.stride(0), lib.ptr(ctx.seq_start), lib.ptr(ctx.slots), nt, ctx.B, H, self.dim, self.rank):
            return
        rec = ctx.scratch("decay.rec", (H, nt, lib.decay_record_size(self.dim)), torch.float32)
        th = ctx.scratch("decay.tanh", (nt, self.tanh_width), self.dtype)
        lib.call("tb_decay_tanh_" + sfx, lib.ptr(a), self.rank, lib.ptr(th), nt, self.rank, self.tanh_width)
        pre = ctx.scratch("decay.pre", (nt, hd), torch.float32)
        matmul_nt(th, w["w2_tanh"], pre)                                    # float out
        lib.call("tb_decay_prep_" + sfx, lib.ptr(z), lib.ptr(pre), lib.ptr(w["w0"]), lib.ptr(w["u"]), lib.ptr(rec),
                 nt, H, self.dim)
        o = ctx.scratch("decay.o", (nt, hd), torch.float32)
        lib.call("tb_decay_scan_" + sfx, lib.ptr(rec), lib.ptr(state), pitch, lib.ptr(o), lib.ptr(x1), d,
                 lib.ptr(ctx.seq_start), lib.ptr(ctx.slots), nt, ctx.B, H, self.dim)
        gate = z[3 * nt:]
        lib.call("tb_mlstm_out_" + sfx, lib.ptr(o), lib.ptr(gate), hd, lib.ptr(w["norm"]), lib.ptr(rows), nt, H, self.dim,
                 self.eps, 1, rows.stride(0))

    def forward(self, ctx, x1, out, cache, state) -> None:
        rows = ctx.scratch("decay.y", (x1.shape[0], self.hd), self.dtype)
        self.forward_rows(ctx, x1, rows, cache, state)
        matmul_nt(rows, self.weights["wo"], out)

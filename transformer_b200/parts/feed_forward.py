"""Feed-forward parts: a dense SwiGLU and a softmax-top-k mixture of SwiGLU experts.

The reference runs the experts as a host loop over tokens and chosen experts with one product
each and a device-to-host copy of the router logits in every layer
(models/llama/common/src/compute.rs:294-333).  Here the tokens are sorted by expert on the device
and every expert runs once over all of its tokens (a grouped product); nothing touches the host.
"""
from __future__ import annotations

import torch

from ..csrc import lib
from .base import FEED_FORWARDS, FeedForward, NormTail, ParamDecl, WeightedRows
from . import linear
from .linear import gemm_skinny, grouped_matmul, matmul_nt

ROUTER_ROWS_FROM = 256      # above this many tokens the router works on tiles of 16 tokens (tensor cores)
ROUTER_TAIL_ROWS = 256      # up to this many tokens the norm before the experts also routes


@FEED_FORWARDS.register("swiglu")
class DenseSwiGLU(FeedForward):
    """params: width, di, bias (default False).  gate_up = x1 Wgu^T (gate rows first), h = silu(gate) * up,
    out = h Wd^T (compute.rs:278-292).  With ``bias`` all three projections have one: ``bgu`` (gate's, then up's)
    and ``bd``, float.  The down projection's bias rides inside its product: the bound weight gets the bias as one
    more column (and zeros up to a multiple of eight), and the kernel that applies the pair's biases and the
    activation writes a one into that column of ``h``.  ``glu_limit`` (with ``glu_alpha``, default 1): the pair
    becomes g' * sigmoid(alpha g') * (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit) instead of
    silu(g) * u, in the product's epilogue.  ``act`` = "gelu_tanh": gelu(g) * u with the tanh form of gelu, there too."""
    graph_safe = True
    launches_only = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.d = int(params["width"])
        self.di = int(params["di"])
        self.bias = bool(params.get("bias", False))
        limit = params.get("glu_limit")
        self.glu = None if limit is None else (float(params.get("glu_alpha", 1.0)), float(limit))
        if self.glu is not None and self.bias:
            raise ValueError("the clamped pair has no form with biases")
        act = params.get("act", "silu")
        if act not in ("silu", linear.GELU_TANH):
            raise ValueError(f"unknown activation {act!r}; this part has 'silu' and 'gelu_tanh'")
        if act != "silu":
            if self.glu is not None or self.bias:
                raise ValueError("the tanh form of gelu goes with neither the clamped pair nor biases")
            self.glu = act

    def parameters(self):
        decl = {"wgu": ParamDecl((2 * self.di, self.d)), "wd": ParamDecl((self.d, self.di))}
        if self.bias:
            decl["bgu"] = ParamDecl((2 * self.di,), "norm", "normal")
            decl["bd"] = ParamDecl((self.d,), "norm", "normal")
        return decl

    def bind(self, tensors) -> None:
        super().bind(tensors)
        if self.bias:
            wd, bd = self.weights["wd"], self.weights.pop("bd")
            pad = (self.di + 1 + 7) // 8 * 8 - self.di - 1
            self.weights["wd"] = torch.cat([wd, bd.to(wd.dtype)[:, None], wd.new_zeros((self.d, pad))], dim=1).contiguous()

    def forward(self, ctx, x1, out) -> None:
        nt = x1.shape[0]
        if self.bias:
            wide = self.weights["wd"].shape[1]
            gu = ctx.scratch("ff.gu", (nt, 2 * self.di), self.dtype)
            matmul_nt(x1, self.weights["wgu"], gu)
            h = ctx.scratch("ff.h1", (nt, wide), self.dtype)
            lib.call("tb_bias_glu_" + lib.suffix(self.dtype), lib.ptr(gu), lib.ptr(self.weights["bgu"]), lib.ptr(h), nt,
                     self.di, wide)
            matmul_nt(h, self.weights["wd"], out)
            return
        h = ctx.scratch("ff.h", (nt, self.di), self.dtype)
        grouped_matmul(x1, self.weights["wgu"], h, swiglu=True, glu=self.glu)
        matmul_nt(h, self.weights["wd"], out)


@FEED_FORWARDS.register("mlp")
class DenseMLP(FeedForward):
    """params: width, di, act ("relu2").  A feed-forward without a gate: out = act(x1 Wu^T) Wd^T, with
    relu2(z) = max(z, 0)^2 (float, one rounding).  The activation sits in the epilogue of this package's own products
    (decoding, and the 32-bit path); behind the library's product of many bfloat16 rows it is a pass of its own over
    the result, in place."""
    graph_safe = True
    launches_only = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.d = int(params["width"])
        self.di = int(params["di"])
        self.act = params.get("act", "relu2")
        if self.act != "relu2":
            raise ValueError(f"unknown activation {self.act!r}; this part has 'relu2'")

    def parameters(self):
        return {"wu": ParamDecl((self.di, self.d)), "wd": ParamDecl((self.d, self.di))}

    def forward(self, ctx, x1, out) -> None:
        nt = x1.shape[0]
        h = ctx.scratch("ff.h", (nt, self.di), self.dtype)
        if self.dtype == torch.float32:
            linear.gemm_simt(x1, self.weights["wu"], h, out_kind=3)
        elif not (nt <= linear.SKINNY_MAX_ROWS and gemm_skinny(x1, self.weights["wu"], h, out_kind=3)):
            matmul_nt(x1, self.weights["wu"], h)
            lib.call("tb_relu2_" + lib.suffix(self.dtype), lib.ptr(h), nt * self.di)
        matmul_nt(h, self.weights["wd"], out)


@FEED_FORWARDS.register("moe")
class MoE(FeedForward):
    """params: width, di, nexp, nexp_use; optional: scoring, correction, identity, glu_alpha, glu_limit.

    router logits (float) -> the nexp_use largest, equal logits to the lower expert -> softmax over
    the kept logits (compute.rs:375-394) -> expert SwiGLU (compute.rs:320-328) -> weighted sum in
    descending-logit order, in float (compute.rs:329-330).

    Other routers and experts, by parameter:
    * ``scoring`` = "all": scores = softmax over ALL router outputs; the nexp_use largest of score + correction
      are chosen (``correction`` = True: a learned float vector, one entry per router output; equal values to the
      lower index); the weights are the chosen scores as they are.
    * ``identity`` = n: the router has nexp + n outputs, and the last n stand for experts without weights whose
      output is their input.
    * ``glu_limit`` (with ``glu_alpha``): the expert's pair becomes g' * sigmoid(alpha g') * (u' + 1) with
      g' = min(g, limit), u' = clamp(u, -limit, limit), instead of silu(g) * u.
    * ``scoring`` = "sigmoid": scores = sigmoid(logit), each by itself; the nexp_use largest are chosen (equal values
      to the lower index); the weights are the chosen scores as they are.
    * ``weight_on`` = "input": the weight multiplies what the expert reads, out = sum_e expert_e(w_e x1), instead of
      what it returns.  Every (token, choice) pair gets its own scaled copy of the token's row (one kernel, which
      also puts the rows in the experts' order), the experts run on those, and their results are summed unweighted.
    * ``scoring`` = "table": no router.  A table (weight ``table``, [vocab, nexp_use] int32, the entries of a row differ)
      gives every token id its experts; every weight is 1 / nexp_use.
    * ``shared_di`` = n: one more expert of width n (weights ``shared_wgu``, ``shared_wd``; ``shared_limit`` and
      ``glu_alpha`` as above), which every token passes; its result is multiplied by sigmoid(gate . x1), one number a
      token (weight ``shared_gate``), and joins the same weighted sum."""
    graph_safe = True
    launches_only = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.d = int(params["width"])
        self.di = int(params["di"])
        self.E = int(params["nexp"])
        self.k = int(params["nexp_use"])
        if not (0 < self.k <= self.E + int(params.get("identity", 0))):
            raise ValueError(f"experts per token {self.k} must lie in 1..{self.E + int(params.get('identity', 0))}")
        self.identity = int(params.get("identity", 0))
        self.R = self.E + self.identity           # router outputs
        if self.R > 1024:
            raise ValueError(f"the routing kernels take up to 1024 experts, got {self.R}")
        self.scoring = params.get("scoring", "kept")
        if self.scoring not in ("kept", "all", "sigmoid", "table"):
            raise ValueError(f"unknown router scoring {self.scoring!r}")
        self.weight_on = params.get("weight_on", "output")
        if self.weight_on not in ("output", "input"):
            raise ValueError(f"the router's weight multiplies the expert's 'output' or 'input', got {self.weight_on!r}")
        if self.weight_on == "input" and self.identity:
            raise ValueError("pass-through experts and weights on the input are not combined")
        self.correction = bool(params.get("correction", False))
        if self.correction and self.scoring != "all":
            raise ValueError("a correction of the choice goes with scoring 'all'")
        limit = params.get("glu_limit")
        self.glu = None if limit is None else (float(params.get("glu_alpha", 1.0)), float(limit))
        self.plain_router = self.scoring == "kept" and not self.identity
        self.table = self.scoring == "table"
        self.vocab = int(params.get("vocab", 0))
        if self.table and (self.identity or self.weight_on == "input" or self.vocab <= 0):
            raise ValueError("a table of experts needs 'vocab' and goes with neither pass-through experts nor weights on the input")
        self.shared = int(params.get("shared_di") or 0)
        if self.shared and (self.identity or self.weight_on == "input"):
            raise ValueError("a shared expert goes with neither pass-through experts nor weights on the input")
        limit = params.get("shared_limit")
        self.shared_glu = None if limit is None else (float(params.get("glu_alpha", 1.0)), float(limit))
        self.terms = self.k + (1 if self.shared else 0)       # of a token's sum

    def parameters(self):
        decl = {
            "wgu": ParamDecl((self.E, 2 * self.di, self.d)),
            "wd": ParamDecl((self.E, self.d, self.di)),
        }
        if self.table:
            decl["table"] = ParamDecl((self.vocab, self.k), "table", f"distinct:{self.E}")
        else:
            decl["router"] = ParamDecl((self.R, self.d))
        if self.shared:
            decl["shared_wgu"] = ParamDecl((2 * self.shared, self.d))
            decl["shared_wd"] = ParamDecl((self.d, self.shared))
            decl["shared_gate"] = ParamDecl((1, self.d))
        if self.correction:
            decl["correction"] = ParamDecl((self.R,), "norm", "normal")
        return decl

    def bind(self, tensors) -> None:
        super().bind(tensors)
        if self.table:
            t = self.weights["table"]
            lo, hi = int(t.min()), int(t.max())
            if lo < 0 or hi >= self.E:
                raise ValueError(f"the table names experts {lo}..{hi}, but there are {self.E}")

    def early_weights(self):
        """The router's matrix: small, and every token's block waits for all of it."""
        r = self.weights.get("router")
        return r if r is not None and r.numel() * r.element_size() <= (1 << 20) else None

    def route(self, ctx, x1, logits_out=None, lists=None):
        """Experts and weights of every token.  With ``lists`` = (offsets, sorted_token, pair_row) the dispatch lists
        are wanted too; returns (idx, w, whether the lists were built along the way)."""
        nt = x1.shape[0]
        idx = ctx.scratch("moe.topk_idx", (nt, self.k), torch.int32)
        w = ctx.scratch("moe.topk_w", (nt, self.k), torch.float32)
        if self.scoring == "all":
            # scores over all outputs, choice with the correction, the block that finishes last builds the lists
            done = ctx.scratch("moe.done", (1,), torch.int32, zero=True) if lists is not None else None
            offsets, sorted_token, pair_row = lists if lists is not None else (None, None, None)
            if self.dtype == torch.bfloat16 and nt > ROUTER_ROWS_FROM and self.R <= 64 and \
                    lib.try_call("tb_router_rows_scored_bf16", lib.ptr(x1), lib.ptr(self.weights["router"]),
                                 lib.ptr(self.weights.get("correction")), lib.ptr(idx), lib.ptr(w), lib.ptr(offsets),
                                 lib.ptr(sorted_token), lib.ptr(pair_row), lib.ptr(done), nt, self.d, self.R, self.k):
                return idx, w, lists is not None
            lib.call("tb_router_scored_" + lib.suffix(self.dtype), lib.ptr(x1), lib.ptr(self.weights["router"]),
                     lib.ptr(self.weights.get("correction")), lib.ptr(idx), lib.ptr(w), lib.ptr(offsets),
                     lib.ptr(sorted_token), lib.ptr(pair_row), lib.ptr(done), nt, self.d, self.R, self.k)
            return idx, w, lists is not None
        if self.scoring == "sigmoid":
            # the same kernels with another rule for the weights; the block that finishes last builds the lists
            done = ctx.scratch("moe.done", (1,), torch.int32, zero=True) if lists is not None else None
            offsets, sorted_token, pair_row = lists if lists is not None else (None, None, None)
            if self.dtype == torch.bfloat16 and nt > ROUTER_ROWS_FROM and self.R <= 64 and \
                    lib.try_call("tb_router_rows_sigmoid_bf16", lib.ptr(x1), lib.ptr(self.weights["router"]),
                                 lib.ptr(idx), lib.ptr(w), lib.ptr(offsets), lib.ptr(sorted_token), lib.ptr(pair_row),
                                 lib.ptr(done), nt, self.d, self.R, self.k):
                return idx, w, lists is not None
            lib.call("tb_router_sigmoid_" + lib.suffix(self.dtype), lib.ptr(x1), lib.ptr(self.weights["router"]),
                     lib.ptr(idx), lib.ptr(w), lib.ptr(offsets), lib.ptr(sorted_token), lib.ptr(pair_row),
                     lib.ptr(done), nt, self.d, self.R, self.k)
            return idx, w, lists is not None
        if self.dtype == torch.bfloat16 and nt > ROUTER_ROWS_FROM and self.R <= 64:
            # many tokens, few experts: 16 tokens' logits are a tensor-core tile, the activations are read once, and
            # the block that finishes last builds the dispatch lists
            done = ctx.scratch("moe.done", (1,), torch.int32, zero=True) if lists is not None else None
            offsets, sorted_token, pair_row = lists if lists is not None else (None, None, None)
            if lib.try_call("tb_router_rows_bf16", lib.ptr(x1), lib.ptr(self.weights["router"]), lib.ptr(idx), lib.ptr(w),
                            lib.ptr(logits_out), lib.ptr(offsets), lib.ptr(sorted_token), lib.ptr(pair_row),
                            lib.ptr(done), nt, self.d, self.R, self.k):
                return idx, w, lists is not None
        # a few tokens: the block that finishes last builds the lists, which saves a kernel on the way to the experts
        fused = lists is not None and nt <= ROUTER_ROWS_FROM
        done = ctx.scratch("moe.done", (1,), torch.int32, zero=True) if fused else None
        offsets, sorted_token, pair_row = lists if fused else (None, None, None)
        lib.call("tb_router_" + lib.suffix(self.dtype), lib.ptr(x1), lib.ptr(self.weights["router"]),
                 lib.ptr(idx), lib.ptr(w), lib.ptr(logits_out), lib.ptr(offsets), lib.ptr(sorted_token),
                 lib.ptr(pair_row), lib.ptr(done), nt, self.d, self.R, self.k)
        return idx, w, fused

    def norm_tail(self, ctx, nt):
        """For a few tokens the router rides along with the norm before this part."""
        if self.table:
            return NormTail("terms", table=self.weights["table"], k=self.k,
                            gate=self.weights["shared_gate"] if self.shared else None,
                            index=ctx.scratch("moe.topk_idx", (nt, self.k), torch.int32),
                            scores=ctx.scratch("moe.terms_w", (nt, self.terms), torch.float32))
        if nt > ROUTER_TAIL_ROWS:
            return None
        return NormTail("router", weights=self.weights["router"], k=self.k,
                        index=ctx.scratch("moe.topk_idx", (nt, self.k), torch.int32),
                        scores=ctx.scratch("moe.topk_w", (nt, self.k), torch.float32),
                        scored=self.scoring == "all", bias=self.weights.get("correction"),
                        sigmoid=self.scoring == "sigmoid")

    def _terms(self, ctx, x1, tail):
        """(experts [nt, k], weights [nt, terms]) of every token's sum, where a table chooses or a shared expert joins."""
        nt = x1.shape[0]
        if tail is not None and tail.kind == "terms":
            return tail.index, tail.scores
        table = self.weights.get("table")
        if table is None:
            idx, w_in = (tail.index, tail.scores) if tail is not None else self.route(ctx, x1)[:2]
        else:
            idx, w_in = ctx.scratch("moe.topk_idx", (nt, self.k), torch.int32), None
        w = ctx.scratch("moe.terms_w", (nt, self.terms), torch.float32)
        lib.call("tb_moe_terms_" + lib.suffix(self.dtype), lib.ptr(x1), lib.ptr(self.weights.get("shared_gate")),
                 lib.ptr(ctx.tok_ids), lib.ptr(table), lib.ptr(w_in), lib.ptr(idx), lib.ptr(w), nt, self.d, self.k)
        return idx, w

    def _shared(self, ctx, x1, out) -> None:
        h = ctx.scratch("moe.shared_h", (x1.shape[0], self.shared), self.dtype)
        grouped_matmul(x1, self.weights["shared_wgu"], h, swiglu=True, glu=self.shared_glu)
        matmul_nt(h, self.weights["shared_wd"], out)

    def _forward_terms(self, ctx, x1, tail):
        """The step where a table chooses the experts or a shared expert joins: the experts' rows and the shared
        expert's lie one behind the other, and all of them are terms of one weighted sum."""
        nt = x1.shape[0]
        M = nt * self.k
        rows = ctx.scratch("moe.y", (M + (nt if self.shared else 0), self.d), self.dtype)
        y = rows[:M]
        idx, w = self._terms(ctx, x1, tail)
        ctx.record("moe.topk_idx", idx)
        h = ctx.scratch("moe.h", (M, self.di), self.dtype)
        at = None
        if self.dtype == torch.bfloat16 and M <= linear.SKINNY_MAX_PAIRS and self.d % 8 == 0 and self.di % 8 == 0:
            pairs = idx.view(-1)
            if gemm_skinny(x1, self.weights["wgu"], h, groups=self.E, out_kind=2, max_group_rows=nt, row_group=pairs,
                           x_div=self.k, glu=self.glu) and \
                    gemm_skinny(h, self.weights["wd"], y, groups=self.E, max_group_rows=nt, row_group=pairs):
                at = _term_rows(nt, self.k, bool(self.shared), x1.device)
        if at is None:
            offsets = ctx.scratch("moe.offsets", (self.E + 1,), torch.int32)
            sorted_token = ctx.scratch("moe.sorted_token", (M,), torch.int32)
            at = ctx.scratch("moe.term_row", (nt * self.terms,), torch.int32)
            lib.call("tb_moe_dispatch_shared" if self.shared else "tb_moe_dispatch", lib.ptr(idx), lib.ptr(offsets),
                     lib.ptr(sorted_token), lib.ptr(at), M, self.k, self.E)
            grouped_matmul(x1, self.weights["wgu"], h, a_rows=sorted_token, group_offsets=offsets, groups=self.E,
                           swiglu=True, max_group_rows=nt, scratch=ctx.scratch, glu=self.glu)
            grouped_matmul(h, self.weights["wd"], y, group_offsets=offsets, groups=self.E, max_group_rows=nt)
        if self.shared:
            self._shared(ctx, x1, rows[M:])
        return WeightedRows(rows, at, w, self.terms)

    def forward(self, ctx, x1, out, tail=None) -> None:
        if self.table or self.shared:
            return self._forward_terms(ctx, x1, tail)
        nt = x1.shape[0]
        M = nt * self.k
        sfx = lib.suffix(self.dtype)
        if self.dtype == torch.bfloat16 and M <= linear.SKINNY_MAX_PAIRS and self.d % 8 == 0 and self.di % 8 == 0:
            # a few tokens: no dispatch lists.  Row p = t * k + j of the experts' products is the pair (token t,
            # its j-th choice); every block of the product kernel finds its expert's pairs in the router's answer
            idx, w = (tail.index, tail.scores) if tail is not None else self.route(ctx, x1)[:2]
            h = ctx.scratch("moe.h", (M, self.di), self.dtype)
            y = ctx.scratch("moe.y", (M, self.d), self.dtype)
            pairs = idx.view(-1)
            src, x_div = x1, self.k
            if self.weight_on == "input":       # a scaled copy of the token's row for each of its pairs
                src, x_div = ctx.scratch("moe.scaled_rows", (M, self.d), self.dtype), 1
                lib.call("tb_moe_scaled_rows_" + sfx, lib.ptr(x1), lib.ptr(w), 0, lib.ptr(src), M, self.d, self.k)
                w = _ones(nt, self.k, x1.device)
            if gemm_skinny(src, self.weights["wgu"], h, groups=self.E, out_kind=2, max_group_rows=nt, row_group=pairs,
                           x_div=x_div, glu=self.glu) and \
                    gemm_skinny(h, self.weights["wd"], y, groups=self.E, max_group_rows=nt, row_group=pairs):
                ctx.record("moe.topk_idx", idx)
                if self.identity:       # pairs that chose an expert without weights: the token's own row
                    lib.call("tb_moe_identity_rows_" + sfx, lib.ptr(x1), lib.ptr(y), 0, 0, lib.ptr(pairs), self.k, M,
                             self.d, self.E)
                return WeightedRows(y, _identity_rows(M, x1.device), w, self.k)
        offsets = ctx.scratch("moe.offsets", (self.R + 1,), torch.int32)
        sorted_token = ctx.scratch("moe.sorted_token", (M,), torch.int32)
        pair_row = ctx.scratch("moe.pair_row", (M,), torch.int32)
        if tail is not None:
            idx, w, listed = tail.index, tail.scores, False
        else:
            idx, w, listed = self.route(ctx, x1, lists=(offsets, sorted_token, pair_row))
        ctx.record("moe.topk_idx", idx)
        if not listed:
            lib.call("tb_moe_dispatch", lib.ptr(idx), lib.ptr(offsets), lib.ptr(sorted_token), lib.ptr(pair_row),
                     M, self.k, self.R)
        h = ctx.scratch("moe.h", (M, self.di), self.dtype)
        if self.weight_on == "input":
            # the pairs' scaled rows, already in the experts' order (what the gather before the product does else)
            src = ctx.scratch("grouped.sorted_rows", (M, self.d), self.dtype)
            lib.call("tb_moe_scaled_rows_" + sfx, lib.ptr(x1), lib.ptr(w), lib.ptr(pair_row), lib.ptr(src), M, self.d,
                     self.k)
            w = _ones(nt, self.k, x1.device)
            grouped_matmul(src, self.weights["wgu"], h, group_offsets=offsets, groups=self.E, swiglu=True,
                           max_group_rows=nt, scratch=ctx.scratch, glu=self.glu)
        else:
            grouped_matmul(x1, self.weights["wgu"], h, a_rows=sorted_token, group_offsets=offsets, groups=self.E,
                           swiglu=True, max_group_rows=nt, scratch=ctx.scratch, glu=self.glu)
        y = ctx.scratch("moe.y", (M, self.d), self.dtype)
        grouped_matmul(h, self.weights["wd"], y, group_offsets=offsets, groups=self.E, max_group_rows=nt)
        if self.identity:               # the rows after the last real expert's: their tokens' own rows
            lib.call("tb_moe_identity_rows_" + sfx, lib.ptr(x1), lib.ptr(y), lib.ptr(offsets), lib.ptr(sorted_token),
                     0, 1, M, self.d, self.E)
        # the weighted sum over the chosen experts is left to the norm that follows (fused there)
        return WeightedRows(y, pair_row, w, self.k)


_IDENTITY_ROWS = {}


def _identity_rows(n: int, device) -> torch.Tensor:
    """0 .. n-1 as int32, made once per size."""
    key = (n, str(device))
    if key not in _IDENTITY_ROWS:
        _IDENTITY_ROWS[key] = torch.arange(n, dtype=torch.int32, device=device)
    return _IDENTITY_ROWS[key]


_TERM_ROWS = {}


def _term_rows(nt: int, k: int, shared: bool, device) -> torch.Tensor:
    """The rows of every token's terms where pair (t, j) lies in row t k + j and a shared expert's results in the rows
    behind, made once per size."""
    if not shared:
        return _identity_rows(nt * k, device)
    key = (nt, k, str(device))
    if key not in _TERM_ROWS:
        pairs = torch.arange(nt * k, dtype=torch.int32).view(nt, k)
        own = nt * k + torch.arange(nt, dtype=torch.int32)
        _TERM_ROWS[key] = torch.cat([pairs, own[:, None]], dim=1).reshape(-1).contiguous().to(device)
    return _TERM_ROWS[key]


_ONES = {}


def _ones(nt: int, k: int, device) -> torch.Tensor:
    """[nt, k] float ones, made once per size: the weights of a sum whose terms were weighted on the way in."""
    key = (nt, k, str(device))
    if key not in _ONES:
        _ONES[key] = torch.ones((nt, k), dtype=torch.float32, device=device)
    return _ONES[key]


def sum_weighted_rows(wr: WeightedRows, out) -> None:
    """out[t] = sum_j weights[t, j] * rows[index[t, j]], for a consumer that wants a plain tensor."""
    nt, d = out.shape
    lib.call("tb_moe_combine_" + lib.suffix(out.dtype), lib.ptr(wr.rows), lib.ptr(wr.index), lib.ptr(wr.weights),
             lib.ptr(out), nt, d, wr.k)

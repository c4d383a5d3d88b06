"""The Fofapel decoder: blocks whose parts read the residual stream as it is and that norm the stream itself behind each
part, x <- LN(alpha x + part(x)).  Every mixer is two side by side: windowed grouped-query attention whose values are
its keys as projected (biases, a norm per head without weights, a sink of score zero, one sigmoid gate per head), and a
linear memory with a decay per key channel made from the input, a bonus for the current token and a shift by one token.
The feed-forward is a dense pair with the tanh form of gelu, or experts that a table chooses by token id beside an expert
that every token passes.

Everything particular to the design lives here: how its configuration becomes a :class:`ModelSpec`, and which
file tensors fill which parameters.  Tensor names of a model file (linear weights [out, in]):

    embed [vocab, width]    final.norm, final.norm.b [width]    head [vocab, width]
    l<i>.norm1, .norm1.b [width]      the norm behind the mixer;  .norm2, .norm2.b behind the feed-forward
    l<i>.mix.left.q [heads dim, width]  .q.b [heads dim]  .k [kv_heads dim, width]  .k.b [kv_heads dim]
                  .g [heads, width]  .o [width, heads dim]
    l<i>.mix.right.mu.r, .mu.k, .mu.v, .mu.g, .mu.w [width]  .r, .k, .v, .g [heads dim, width]  .w1 [rank, width]
                  .w2 [heads dim, rank]  .w0 [heads dim]  .u [heads, dim]  .norm [heads dim]  .o [width, heads dim]
    dense:        l<i>.mlp.gate, .up [ff, width]  .down [width, ff]
    moe:          l<i>.mlp.e<j>.gate, .e<j>.up [ff, width]  .e<j>.down [width, ff]  .table [vocab, top] (integers)
                  .shared.gate, .shared.up, .shared.down alike with the shared width  .shared.sg [1, width]
"""
from __future__ import annotations

from typing import List

from ..config.fofapel import DenseMeta, FofapelMeta
from ..config.registry import Architecture, ConfigError, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..weights.plan import Source, TensorRule, single

GLU_ALPHA = 1.702       # the slope inside the clamped pair's sigmoid
SINK = 0.0              # the score that joins every softmax without a value


def _rank(x, where) -> int:
    if x.decay_rank is None:
        raise ConfigError(f"{where}: the rank of the decay's projections is known neither from the configuration "
                          f"(decay_rank) nor from a weight file")
    return x.decay_rank


def build_spec(m: FofapelMeta) -> ModelSpec:
    norm = PartSpec.of("layernorm", width=m.width, eps=m.eps, bias=True, stream=m.alpha)
    layers = []
    for i, layer in enumerate(m.layers):
        a, r = layer.mixer.left, layer.mixer.right
        rope = PartSpec.of("rope", dh=a.rot_dims, theta=a.rot_base, pairing="adjacent", positions=m.max_context)
        left = PartSpec.of("attention", width=m.width, nh=a.heads, nkvh=a.kv_heads, dh=a.dim, scale=a.scale,
                           window=a.window, values="keys", bias=True, qk_norm="unit", eps=m.eps, head_gate=True,
                           sink_value=SINK, out_scale=layer.mixer.left_scale, position=rope if a.rot_dims else None)
        right = PartSpec.of("decay_memory", width=m.width, heads=r.heads, dim=r.dim,
                            rank=_rank(r, f"layers[{i}].mixer.right"), eps=m.eps, out_scale=layer.mixer.right_scale)
        f, ff = layer.mlp, None
        if isinstance(f, DenseMeta):
            ff = PartSpec.of("swiglu", width=m.width, di=f.ff, act="gelu_tanh")
        elif f is not None:
            shared = {} if f.shared is None else {"shared_di": f.shared.ff, "shared_limit": f.shared.limit}
            ff = PartSpec.of("moe", width=m.width, di=f.expert.ff, nexp=f.experts, nexp_use=f.top, scoring="table",
                             vocab=m.vocab, glu_alpha=GLU_ALPHA, glu_limit=f.expert.limit, **shared)
        layers.append(LayerSpec(mixer=PartSpec.of("side_by_side", width=m.width, left=left, right=right), feed_forward=ff,
                                mixer_norm=norm, feed_forward_norm=None if ff is None else norm,
                                arrangement="post_norm"))
    return ModelSpec(
        width=m.width, vocab=m.vocab, max_context=m.max_context, layers=tuple(layers),
        order=tuple(RunEntry(i) for i in range(len(layers))),
        embedding=PartSpec.of("lookup", vocab=m.vocab, width=m.width),
        final_norm=PartSpec.of("layernorm", width=m.width, eps=m.eps, bias=True),
        head=PartSpec.of("linear", vocab=m.vocab, width=m.width, tied=False),
        stop_tokens=tuple(m.eos),
    )


def tensor_plan(m: FofapelMeta) -> List[TensorRule]:
    d = m.width
    rules = [TensorRule(("embedding", "table"), (m.vocab, d), "matrix", (single("embed", (m.vocab, d)),))]
    for i, layer in enumerate(m.layers):
        p, L = f"l{i}.", ("layers", i)
        mx = L + ("mixer",)

        def vec(dest, name, shape, init="normal"):
            rules.append(TensorRule(dest, tuple(shape), "norm", (single(p + name, shape),), init=init))

        def mat(dest, name, shape):
            rules.append(TensorRule(dest, tuple(shape), "matrix", (single(p + name, shape),)))

        def joined(dest, shape, names, shapes, how, role="matrix"):
            rules.append(TensorRule(dest, tuple(shape), role, (Source(tuple(p + n for n in names), tuple(shapes), how),)))

        def norm(part, n):
            vec(L + (part, "weight"), f"norm{n}", (d,), "ones")
            vec(L + (part, "bias"), f"norm{n}.b", (d,))

        norm("mixer_norm", 1)
        a, r = layer.mixer.left, layer.mixer.right
        hq, hk = a.heads * a.dim, a.kv_heads * a.dim
        joined(mx + ("left.wqkv",), (hq + hk + a.heads, d), ("mix.left.q", "mix.left.k", "mix.left.g"),
               ((hq, d), (hk, d), (a.heads, d)), "cat0")
        joined(mx + ("left.bqk",), (hq + hk,), ("mix.left.q.b", "mix.left.k.b"), ((hq,), (hk,)), "cat0", "norm")
        mat(mx + ("left.wo",), "mix.left.o", (d, hq))
        hd, rank = r.heads * r.dim, _rank(r, f"layers[{i}].mixer.right")
        joined(mx + ("right.mu",), (5, d), tuple(f"mix.right.mu.{c}" for c in "rkvgw"), ((d,),) * 5, "stack0", "norm")
        joined(mx + ("right.win",), (4, hd, d), tuple(f"mix.right.{c}" for c in "rkvg"), ((hd, d),) * 4, "stack0")
        mat(mx + ("right.w1",), "mix.right.w1", (rank, d))
        mat(mx + ("right.w2",), "mix.right.w2", (hd, rank))
        vec(mx + ("right.w0",), "mix.right.w0", (hd,))
        vec(mx + ("right.u",), "mix.right.u", (r.heads, r.dim))
        vec(mx + ("right.norm",), "mix.right.norm", (hd,), "ones")
        mat(mx + ("right.wo",), "mix.right.o", (d, hd))
        f = layer.mlp
        if f is None:
            continue
        norm("feed_forward_norm", 2)
        ff = L + ("feed_forward",)
        if isinstance(f, DenseMeta):
            joined(ff + ("wgu",), (2 * f.ff, d), ("mlp.gate", "mlp.up"), ((f.ff, d),) * 2, "cat0")
            mat(ff + ("wd",), "mlp.down", (d, f.ff))
            continue
        E, n = f.experts, f.expert.ff
        joined(ff + ("wgu",), (E, 2 * n, d), tuple(f"mlp.e{e}.{which}" for e in range(E) for which in ("gate", "up")),
               ((n, d),) * (2 * E), "stack0_of_row_pairs")
        joined(ff + ("wd",), (E, d, n), tuple(f"mlp.e{e}.down" for e in range(E)), ((d, n),) * E, "stack0")
        rules.append(TensorRule(ff + ("table",), (m.vocab, f.top), "table", (single(p + "mlp.table", (m.vocab, f.top)),),
                                init=f"distinct:{E}"))
        if f.shared is not None:
            n = f.shared.ff
            joined(ff + ("shared_wgu",), (2 * n, d), ("mlp.shared.gate", "mlp.shared.up"), ((n, d),) * 2, "cat0")
            mat(ff + ("shared_wd",), "mlp.shared.down", (d, n))
            mat(ff + ("shared_gate",), "mlp.shared.sg", (1, d))
    rules.append(TensorRule(("final_norm", "weight"), (d,), "norm", (single("final.norm", (d,)),), init="ones"))
    rules.append(TensorRule(("final_norm", "bias"), (d,), "norm", (single("final.norm.b", (d,)),)))
    rules.append(TensorRule(("head", "weight"), (m.vocab, d), "matrix", (single("head", (m.vocab, d)),)))
    return rules


FOFAPEL = register_architecture(Architecture(
    name="fofapel",
    config_cls=FofapelMeta,
    build_spec=build_spec,
    tensor_plan=tensor_plan,
    names=("fofapel", "Fofapel"),
    refine=lambda m, shapes: m.with_tensor_shapes(shapes),
))

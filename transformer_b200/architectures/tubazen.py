"""The Tubazen decoder: pre-norm blocks whose norm computes no statistics (tanh(alpha x) w + b), whose parts' results pass
a gate of their own before they join the stream, and whose output is averaged with the embedding output and the outputs
of all layers before.  Learned positions are added to the embedding.  Mixers: a gated linear attention, or two mixers side
by side, attention with a learned bias per (distance bucket, head), biases on all projections, a query multiplier that
grows with the position and an output gate, and a delta rule with a decay, a removal rate and a key of its own.

Everything particular to the design lives here: how its configuration becomes a :class:`ModelSpec`, and which
file tensors fill which parameters.  Tensor names of a model file (linear weights [out, in]):

    embed [vocab, width]    pos [max_positions, width]    head [vocab, width]
    a norm:       <name> [width]  <name>.b [width]  <name>.alpha []         embed.norm, final.norm, l<i>.norm1, l<i>.norm2
    l<i>.rg1, .rg2 [width, width]  .rg1.b, .rg2.b [width]    the gates of the mixer's and the feed-forward's result
    l<i>.dwa [i + 2]                                         weights of the embedding output and of layers 0 .. i
    gla:          l<i>.mix.q, .k [heads dim, width]  .v, .g [heads vdim, width]  .o [width, heads vdim]  .norm [vdim]
                  .a1 [rank, width]  .a2 [heads dim, rank]  .a2.b [heads dim]
    parallel:     l<i>.mix.left.q [heads dim, width]  .k [kv_heads dim, width]  .v [kv_heads vdim, width]  their .b
                  .g [heads vdim, width]  .rel [buckets, heads]  .o [width, heads vdim]  .o.b [width]
                  l<i>.mix.right.r, .k, .v, .g, .a [heads dim, width]  .a.b [heads dim]  .w1 [rank, width]
                  .w2 [heads dim, rank]  .w0 [heads dim]  .norm [heads dim]  .o [width, heads dim]
    dense:        l<i>.mlp.gate, .up [ff, width]  .down [width, ff]
"""
from __future__ import annotations

from typing import List

from ..config.registry import Architecture, ConfigError, register_architecture
from ..config.tubazen import GlaMeta, TubazenMeta
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..weights.plan import Source, TensorRule, single


def _known(v, what) -> int:
    if v is None:
        raise ConfigError(f"{what} is known neither from the configuration nor from a weight file")
    return v


def _gla_rank(m, i):
    return _known(m.decay_rank, f"layers[{i}].mixer: the rank of the decay's projections (decay_rank)")


def _right_rank(m, i):
    return _known(m.right.decay_rank, f"layers[{i}].mixer.right: the rank of the decay's projections (decay_rank)")


def _bias_rows(m, i):
    return _known(m.left.bias_rows, f"layers[{i}].mixer.left: the number of distance buckets (bias_rows)")


def build_spec(m: TubazenMeta) -> ModelSpec:
    norm = PartSpec.of("tanh_norm", width=m.width)
    gate = PartSpec.of("sigmoid", width=m.width)
    layers = []
    for i, layer in enumerate(m.layers):
        x = layer.mixer
        if isinstance(x, GlaMeta):
            mixer = PartSpec.of("gated_linear", width=m.width, heads=x.heads, dim=x.dim, vdim=x.vdim, tau=x.tau,
                                rank=_gla_rank(x, i), eps=m.eps)
        else:
            a, r = x.left, x.right
            temp = {"query_temp": (a.temp_coef, a.temp_every)} if a.temp_every else {}
            left = PartSpec.of("attention", width=m.width, nh=a.heads, nkvh=a.kv_heads, dh=a.dim, dv=a.vdim, scale=a.scale,
                               bias=True, out_bias=True, gate=True, positions=m.max_positions,
                               distance_bias=(_bias_rows(x, i), a.bias_max), out_scale=x.left_scale, **temp)
            right = PartSpec.of("split_delta", width=m.width, heads=r.heads, dim=r.dim, rank=_right_rank(x, i), eps=m.eps,
                                out_scale=x.right_scale)
            mixer = PartSpec.of("side_by_side", width=m.width, left=left, right=right)
        extra, ff = [("mixer_residual_gate", gate)], None
        if layer.ff is not None:
            ff = PartSpec.of("swiglu", width=m.width, di=layer.ff, act="gelu_tanh")
            extra.append(("feed_forward_residual_gate", gate))
        layers.append(LayerSpec(mixer=mixer, feed_forward=ff, mixer_norm=norm, feed_forward_norm=None if ff is None else norm,
                                arrangement="pre_norm", extra=tuple(extra)))
    n = len(layers)
    return ModelSpec(
        width=m.width, vocab=m.vocab, max_context=m.max_positions, layers=tuple(layers),
        order=tuple(RunEntry(i, joint=i - 1 if i else None) for i in range(n)),
        joints=tuple(PartSpec.of("depth_average", width=m.width, terms=i + 2) for i in range(n)), last_joint=n - 1,
        embedding=PartSpec.of("positional_lookup", vocab=m.vocab, width=m.width, positions=m.max_positions, norm=norm),
        final_norm=norm,
        head=PartSpec.of("linear", vocab=m.vocab, width=m.width, tied=False, scale=m.logit_scale),
        stop_tokens=tuple(m.eos),
    )


def tensor_plan(m: TubazenMeta) -> List[TensorRule]:
    d = m.width
    rules = []

    def vec(dest, name, shape, init="normal"):
        rules.append(TensorRule(dest, tuple(shape), "norm", (single(name, shape),), init=init))

    def mat(dest, name, shape):
        rules.append(TensorRule(dest, tuple(shape), "matrix", (single(name, shape),)))

    def norm(dest, name, prefix=""):
        vec(dest + (prefix + "weight",), name, (d,), "ones")
        vec(dest + (prefix + "bias",), name + ".b", (d,))
        vec(dest + (prefix + "alpha",), name + ".alpha", (), "ones")

    mat(("embedding", "table"), "embed", (m.vocab, d))
    mat(("embedding", "positions"), "pos", (m.max_positions, d))
    norm(("embedding",), "embed.norm", "norm.")
    for i, layer in enumerate(m.layers):
        p, L = f"l{i}.", ("layers", i)
        mx = L + ("mixer",)

        def joined(dest, names, shapes, how="cat0", role="matrix", shape=None):
            if shape is None:
                shape = (sum(s[0] for s in shapes),) + tuple(shapes[0][1:])
            rules.append(TensorRule(dest, tuple(shape), role, (Source(tuple(p + n for n in names), tuple(shapes), how),)))

        def gate(part, name):
            mat(L + (part, "weight"), p + name, (d, d))
            vec(L + (part, "bias"), p + name + ".b", (d,))

        norm(L + ("mixer_norm",), p + "norm1")
        gate("mixer_residual_gate", "rg1")
        x = layer.mixer
        if isinstance(x, GlaMeta):
            hk, hv, rank = x.heads * x.dim, x.heads * x.vdim, _gla_rank(x, i)
            joined(mx + ("win",), ("mix.q", "mix.k", "mix.v", "mix.g"), ((hk, d), (hk, d), (hv, d), (hv, d)))
            mat(mx + ("a1",), p + "mix.a1", (rank, d))
            mat(mx + ("a2",), p + "mix.a2", (hk, rank))
            vec(mx + ("a2_bias",), p + "mix.a2.b", (hk,))
            vec(mx + ("norm",), p + "mix.norm", (x.vdim,), "ones")
            mat(mx + ("wo",), p + "mix.o", (d, hv))
        else:
            a, r = x.left, x.right
            hq, hk, hv, ho = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, a.heads * a.vdim
            joined(mx + ("left.wqkv",), tuple(f"mix.left.{c}" for c in "qkvg"), ((hq, d), (hk, d), (hv, d), (ho, d)))
            joined(mx + ("left.bqkv",), tuple(f"mix.left.{c}.b" for c in "qkv"), ((hq,), (hk,), (hv,)), role="norm")
            vec(mx + ("left.rel",), p + "mix.left.rel", (_bias_rows(x, i), a.heads))
            mat(mx + ("left.wo",), p + "mix.left.o", (d, ho))
            vec(mx + ("left.bo",), p + "mix.left.o.b", (d,))
            hd, rank = r.heads * r.dim, _right_rank(x, i)
            joined(mx + ("right.win",), tuple(f"mix.right.{c}" for c in "rkvg"), ((hd, d),) * 4)
            joined(mx + ("right.wa",), ("mix.right.a", "mix.right.w1"), ((hd, d), (rank, d)))
            vec(mx + ("right.ba",), p + "mix.right.a.b", (hd,))
            mat(mx + ("right.w2",), p + "mix.right.w2", (hd, rank))
            vec(mx + ("right.w0",), p + "mix.right.w0", (hd,))
            vec(mx + ("right.norm",), p + "mix.right.norm", (hd,), "ones")
            mat(mx + ("right.wo",), p + "mix.right.o", (d, hd))
        if layer.ff is not None:
            norm(L + ("feed_forward_norm",), p + "norm2")
            gate("feed_forward_residual_gate", "rg2")
            joined(L + ("feed_forward", "wgu"), ("mlp.gate", "mlp.up"), ((layer.ff, d),) * 2)
            mat(L + ("feed_forward", "wd"), p + "mlp.down", (d, layer.ff))
        else:       # what belongs to a feed-forward may be in the file or not
            for name, shape in (("norm2", (d,)), ("norm2.b", (d,)), ("norm2.alpha", ()), ("rg2", (d, d)), ("rg2.b", (d,))):
                rules.append(TensorRule(L + ("unused", name), shape, "norm", (single(p + name, shape),), unused=True))
        vec(("joints", i, "weight"), p + "dwa", (i + 2,), "ones")
    norm(("final_norm",), "final.norm")
    mat(("head", "weight"), "head", (m.vocab, d))
    return rules


TUBAZEN = register_architecture(Architecture(
    name="tubazen",
    config_cls=TubazenMeta,
    build_spec=build_spec,
    tensor_plan=tensor_plan,
    names=("tubazen", "Tubazen"),
    refine=lambda m, shapes: m.with_tensor_shapes(shapes),
))

"""Zanelorn: configuration -> model description.

A decoder without a position table, a 32-bit residual stream that starts as a multiple of the embedded rows, and layers whose
branches read the residual itself and whose results alone are normed (arrangement "output_norm" with "norm_scale" joins):
x <- x + m n1(mixer(x)); x <- x + m n2(ff(x)); x <- x + m ns(side(x)), RMS norms with plain weights and one constant m.  Two
mixers, in any order:

* "retention": ``parts.retention.RetentionMixer``, linear attention with rotated queries and keys and a constant decay per head;
* "parallel": ``parts.projected.ParallelMixer`` of a ``parts.attention.RotaryAttention`` (biases, an RMS norm per query and key
  head before the rotation, linearly scaled frequencies, a window whose first tokens stay visible, an output gate) and a
  ``parts.ssm.MambaMixer``, each times a constant.

The feed-forward is dense (exact gelu), a mixture of clamped experts (scores by a softmax over all outputs, a correction for the
choice alone, weights that are not renormalised, identity experts, a gated shared expert), or absent.  ``side`` is
``parts.side.TokenSideBranch``: a part of a second table's row of the token, per layer.  The head is a matrix of its own.

Tensor names: embed, side.embed, head, final.norm; l<i>.{norm1,norm2}; retention: l<i>.mix.{q,k,v,g,o}; parallel:
l<i>.mix.left.{q,q.b,k,k.b,v,v.b,q.norm,k.norm,g,o}, l<i>.mix.right.{in,conv,conv.b,x,dt,dt.b,A_log,D,o};
l<i>.mlp.{up,down} or l<i>.mlp.{router,correction,e<j>.{gate,up,down},shared.{gate,up,down,sg}}; l<i>.side.{gate,proj,norm};
matrices are stored [out, in].
"""
from __future__ import annotations

import math

from ..config.base import register_architecture
from ..config.zanelorn import DenseSizes, RetentionSizes, ZanelornConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, WeightRef

SIGMOID_FACTOR = 1.702       # the design's factor inside the experts' sigmoid


def build_zanelorn_spec(cfg: ZanelornConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    std = 1.0 / math.sqrt(D)

    def join(name):
        return PartSpec("norm_scale", dict(hidden_size=D, eps=eps, scaled=False, factor=cfg.residual_mult),
                        {"weight": WeightRef((name,), init=("uniform", 0.5, 1.5))})

    def scaling(rot):
        return None if rot.factor is None else {"factor": rot.factor}

    def matrix(name, n_in):
        return WeightRef((name,), init=("normal", 1.0 / math.sqrt(n_in)))

    def retention(s, m):
        w = {f"{c}_weight": matrix(m + c, D) for c in "qkvg"}
        w["out_weight"] = matrix(m + "o", s.heads * s.vdim)
        return PartSpec("retention", dict(hidden_size=D, num_heads=s.heads, head_dim=s.dim, v_head_dim=s.vdim, decay=s.decay, norm_eps=eps,
                                          rot_dims=s.rot.dims, rot_base=s.rot.base, rot_scaling=scaling(s.rot)), w)

    def parallel(s, m):
        a, r = s.left, s.right
        w = {f"left.{c}_weight": matrix(f"{m}left.{c}", D) for c in "qkvg"}
        w.update({f"left.{c}_bias": WeightRef((f"{m}left.{c}.b",), init=("normal", 0.3)) for c in "qkv"})
        w.update({f"left.{c}_norm": WeightRef((f"{m}left.{c}.norm",), init=("uniform", 0.5, 1.5)) for c in "qk"})
        w["left.out_weight"] = matrix(m + "left.o", a.heads * a.vdim)
        w.update({"right.in_proj": matrix(m + "right.in", D),
                  "right.conv_weight": matrix(m + "right.conv", r.conv), "right.conv_bias": WeightRef((m + "right.conv.b",), init=("normal", 0.1)),
                  "right.x_proj": matrix(m + "right.x", r.inner),
                  "right.dt_weight": matrix(m + "right.dt", r.dt_rank), "right.dt_bias": WeightRef((m + "right.dt.b",), init=("uniform", -5.0, -1.0)),
                  "right.A_log": WeightRef((m + "right.A_log",), init=("uniform", 0.0, 2.5)),
                  "right.D": WeightRef((m + "right.D",), init=("uniform", 0.5, 1.5)),
                  "right.out_weight": matrix(m + "right.o", r.inner)})
        branches = [dict(name="left", kind="rotary_attention",
                         params=dict(hidden_size=D, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim,
                                     scale=a.scale, norm_eps=eps, qk_norm=False, head_norm="weighted", rot_dims=a.rot.dims,
                                     rot_base=a.rot.base, rot_interleaved=False, rot_scaling=scaling(a.rot), window=a.window,
                                     keep_first=a.keep_first, bias=True, out_gate=True)),
                    dict(name="right", kind="mamba",
                         params=dict(hidden_size=D, inner=r.inner, state_size=r.state, dt_rank=r.dt_rank, conv_taps=r.conv))]
        return PartSpec("parallel", dict(branches=branches, scales=[s.left_scale, s.right_scale]), w)

    def feed_forward(mlp, f):
        if isinstance(mlp, DenseSizes):
            return PartSpec("mlp", dict(hidden_size=D, inner_size=mlp.ff, activation="gelu_erf", bias=False),
                            {"fc_weight": matrix(f + "up", D), "proj_weight": matrix(f + "down", mlp.ff)})
        w = {"router": matrix(f + "router", D), "correction": WeightRef((f + "correction",), init=("normal", 0.02))}
        for e in range(mlp.experts):
            w.update({f"expert{e}.gate": matrix(f"{f}e{e}.gate", D), f"expert{e}.up": matrix(f"{f}e{e}.up", D),
                      f"expert{e}.down": matrix(f"{f}e{e}.down", mlp.ff)})
        if mlp.shared_ff is not None:
            w.update({"shared.gate": matrix(f + "shared.gate", D), "shared.up": matrix(f + "shared.up", D),
                      "shared.down": matrix(f + "shared.down", mlp.shared_ff), "shared.sg": matrix(f + "shared.sg", D)})
        return PartSpec("moe", dict(hidden_size=D, num_experts=mlp.experts, top=mlp.top, expert_size=mlp.ff, identity=mlp.identity,
                                    shared_size=mlp.shared_ff, shared_gate=mlp.shared_ff is not None, activation="swiglu_clamp",
                                    limit=mlp.limit, shared_limit=mlp.shared_limit, alpha=SIGMOID_FACTOR, correction=True, renorm=False), w)

    layers, ignored = [], []
    for i, lay in enumerate(cfg.layers):
        p = f"l{i}."
        mixer = retention(lay.mixer, p + "mix.") if isinstance(lay.mixer, RetentionSizes) else parallel(lay.mixer, p + "mix.")
        ff = None if lay.mlp is None else feed_forward(lay.mlp, p + "mlp.")
        if ff is None:
            ignored.append(rf"^l{i}\.norm2$")        # a layer without a feed-forward has no use for it
        side = PartSpec("gated", dict(hidden_size=D, dim=cfg.side_dim, part=i),
                        {"gate_weight": matrix(p + "side.gate", D), "proj_weight": matrix(p + "side.proj", cfg.side_dim)})
        layers.append(LayerSpec(mixer=mixer, ff=ff, mixer_norm=None, ff_norm=None, arrangement="output_norm", mixer_join=join(p + "norm1"),
                                ff_join=join(p + "norm2") if ff else None, side=side, side_join=join(p + "side.norm")))
    return ModelSpec(hidden_size=D, vocab_size=cfg.vocab,
                     embedding=PartSpec("token", dict(hidden_size=D, vocab_size=cfg.vocab, scale=cfg.embedding_scale, act_copy=True),
                                        {"table": WeightRef(("embed",), init=("normal", 1.0))}),
                     positions=PartSpec("none", {}, {}),
                     token_table=PartSpec("side", dict(vocab_size=cfg.vocab, parts=len(cfg.layers), dim=cfg.side_dim),
                                          {"table": WeightRef(("side.embed",), init=("normal", 1.0))}),
                     layers=layers,
                     final_norm=PartSpec("rmsnorm", dict(hidden_size=D, eps=eps),
                                         {"weight": WeightRef(("final.norm",), init=("uniform", 0.5, 1.5))}),
                     head=PartSpec("linear", dict(hidden_size=D, vocab_size=cfg.vocab), {"weight": WeightRef(("head",), init=("normal", std))}),
                     max_positions=cfg.max_positions, eos_token_id=cfg.eos_token_id, ignored_tensors=ignored)


register_architecture("Zanelorn", ZanelornConfig, build_zanelorn_spec, replace=True)

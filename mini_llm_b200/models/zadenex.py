"""Zadenex: configuration -> model description.

A decoder without a position table, a 32-bit residual stream that starts as a multiple of the embedded rows, and layers
x <- x + m * norm1b(mixer(norm1(x))), x <- x + m * norm2b(ff(norm2(x))): RMS norms with plain weights before and after each
branch and one factor m on the normed result (arrangement "sandwich" with "norm_scale" joins).  Three mixers, in any order:

* "attention": ``parts.attention.MixedScoreAttention``, grouped heads with biases on all four projections, no positions,
  scores mixed over the heads by a matrix, a window, a sink whose score is 0;
* "latent_attention": ``parts.latent.LatentAttention`` with queries through a latent of their own, a rotation of
  neighbouring entries, a sink and a gate per head;
* "mlstm": ``parts.mlstm.MatrixMemoryMixer``, a matrix memory with exponential gates kept below a running maximum.

The feed-forward is gated and dense (the tanh form of gelu) with biases, or absent.  A stretch of layers may run several
times with the same weights; every pass has its own caches and states and begins with x <- W [x; x_0] + (the pass's vector),
x_0 the embedded rows (``parts.passes.PassInput``).  The head is a matrix of its own.

Tensor names: embed, head, final.norm, loop.in, loop.step; l<i>.{norm1,norm1b,norm2,norm2b}; attention:
l<i>.mix.{q,k,v,o}, l<i>.mix.{q,k,v,o}.b, l<i>.mix.talk; latent_attention: l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,g,o};
mlstm: l<i>.mix.{q,k,v,g,i,i.b,f,f.b,norm,o}; l<i>.mlp.{gate,up,down}, l<i>.mlp.{gate,up,down}.b; matrices are stored
[out, in].
"""
from __future__ import annotations

import math

from ..config.base import register_architecture
from ..config.zadenex import AttentionSizes, LatentSizes, ZadenexConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, WeightRef

DENOM_EPS = 1e-6         # the design's addend to the denominator of the matrix memory's output


def build_zadenex_spec(cfg: ZadenexConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    std = 1.0 / math.sqrt(D)

    def norm(name):
        return PartSpec("rmsnorm", dict(hidden_size=D, eps=eps), {"weight": WeightRef((name,), init=("uniform", 0.5, 1.5))})

    def join(name):
        return PartSpec("norm_scale", dict(hidden_size=D, eps=eps, scaled=False, factor=cfg.residual_mult),
                        {"weight": WeightRef((name,), init=("uniform", 0.5, 1.5))})

    layers, ignored = [], []
    for i, lay in enumerate(cfg.layers):
        p = f"l{i}."
        m = p + "mix."
        s = lay.mixer
        if isinstance(s, AttentionSizes):
            w = {f"{c}_weight": WeightRef((m + c,), init=("normal", std)) for c in "qkv"}
            w.update({f"{c}_bias": WeightRef((f"{m}{c}.b",), init=("normal", 0.3)) for c in "qkv"})
            w.update({"talk": WeightRef((m + "talk",), init=("normal", 1.0 / math.sqrt(s.heads))),
                      "out_weight": WeightRef((m + "o",), init=("normal", 1.0 / math.sqrt(s.heads * s.vdim))),
                      "out_bias": WeightRef((m + "o.b",), init=("normal", 0.1))})
            mixer = PartSpec("mixed_score_attention",
                             dict(hidden_size=D, num_heads=s.heads, num_kv_heads=s.kv_heads, head_dim=s.dim, v_head_dim=s.vdim,
                                  scale=s.scale, window=s.window, bias=True, out_bias=True, sink="zero"), w)
        elif isinstance(s, LatentSizes):
            w = {"dq_weight": WeightRef((m + "dq",), init=("normal", std)),
                 "dq_norm": WeightRef((m + "dq.norm",), init=("uniform", 0.5, 1.5)),
                 "uq_weight": WeightRef((m + "uq",), init=("normal", 1.0 / math.sqrt(s.q_rank))),
                 "dkv_weight": WeightRef((m + "dkv",), init=("normal", std)),
                 "dkv_norm": WeightRef((m + "dkv.norm",), init=("uniform", 0.5, 1.5)),
                 "uk_weight": WeightRef((m + "uk",), init=("normal", 1.0 / math.sqrt(s.kv_rank))),
                 "uv_weight": WeightRef((m + "uv",), init=("normal", 1.0 / math.sqrt(s.kv_rank))),
                 "sink": WeightRef((m + "sink",), init=("normal", 1.0)),
                 "g_weight": WeightRef((m + "g",), init=("normal", std)),
                 "out_weight": WeightRef((m + "o",), init=("normal", 1.0 / math.sqrt(s.heads * s.vdim)))}
            mixer = PartSpec("latent_attention",
                             dict(hidden_size=D, num_heads=s.heads, head_dim=s.dim, rot_dim=s.rot_dim, v_head_dim=s.vdim,
                                  kv_rank=s.kv_rank, scale=s.scale, norm_eps=eps, rot_dims=s.rot_dims, rot_base=s.rot_base,
                                  rot_interleaved=True, q_rank=s.q_rank, gate="head", sink=True), w)
        else:
            w = {f"{c}_weight": WeightRef((m + c,), init=("normal", std)) for c in "qkvg"}
            w.update({"i_weight": WeightRef((m + "i",), init=("normal", std)), "i_bias": WeightRef((m + "i.b",), init=("normal", 1.0)),
                      "f_weight": WeightRef((m + "f",), init=("normal", std)), "f_bias": WeightRef((m + "f.b",), init=("uniform", 0.0, 6.0)),
                      "norm_weight": WeightRef((m + "norm",), init=("uniform", 0.5, 1.5)),
                      "out_weight": WeightRef((m + "o",), init=("normal", 1.0 / math.sqrt(s.heads * s.vdim)))})
            mixer = PartSpec("matrix_memory", dict(hidden_size=D, num_heads=s.heads, head_dim=s.dim, v_head_dim=s.vdim,
                                                   gate_cap=s.gate_cap, norm_eps=eps, denom_eps=DENOM_EPS), w)
        ff = None
        if lay.mlp is not None:
            w = {f"{c}_weight": WeightRef((f"{p}mlp.{c}",), init=("normal", std)) for c in ("gate", "up")}
            w["down_weight"] = WeightRef((p + "mlp.down",), init=("normal", 1.0 / math.sqrt(lay.mlp.ff)))
            w.update({f"{c}_bias": WeightRef((f"{p}mlp.{c}.b",), init=("normal", 0.1)) for c in ("gate", "up", "down")})
            ff = PartSpec("gated_mlp", dict(hidden_size=D, inner_size=lay.mlp.ff, activation="gelu_tanh", bias=True), w)
        else:
            ignored.append(rf"^l{i}\.norm2b?$")      # a layer without a feed-forward has no use for them
        layers.append(LayerSpec(mixer=mixer, ff=ff, mixer_norm=norm(p + "norm1"), ff_norm=norm(p + "norm2") if ff else None,
                                arrangement="sandwich", mixer_join=join(p + "norm1b"), ff_join=join(p + "norm2b") if ff else None))
    # a layer's first run keeps the layer's own cache; every further run of a looped layer gets one of its own
    seen, schedule = set(), []
    for li, t in cfg.layer_runs():
        schedule.append(ScheduleEntry(li, private_cache=li in seen, enters_pass=t))
        seen.add(li)
    pass_input = None
    if cfg.loop is not None:
        pass_input = PartSpec("concat_embedding", dict(hidden_size=D, passes=cfg.loop.times),
                              {"weight": WeightRef(("loop.in",), init=("normal", 1.0 / math.sqrt(2 * D))),
                               "step": WeightRef(("loop.step",), init=("normal", 0.5))})
    return ModelSpec(hidden_size=D, vocab_size=cfg.vocab,
                     embedding=PartSpec("token", dict(hidden_size=D, vocab_size=cfg.vocab, scale=cfg.embedding_scale,
                                                      keep=cfg.loop is not None),
                                        {"table": WeightRef(("embed",), init=("normal", 1.0))}),
                     positions=PartSpec("none", {}, {}),
                     layers=layers, final_norm=norm("final.norm"),
                     head=PartSpec("linear", dict(hidden_size=D, vocab_size=cfg.vocab),
                                   {"weight": WeightRef(("head",), init=("normal", std))}),
                     schedule=schedule, pass_input=pass_input, max_positions=cfg.max_positions, eos_token_id=cfg.eos_token_id,
                     ignored_tensors=ignored)


register_architecture("Zadenex", ZadenexConfig, build_zadenex_spec, replace=True)

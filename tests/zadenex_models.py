"""Small Zadenex configurations and weights for the tests: models that differ from each other in every size and option,
with weights that make faults show."""
from __future__ import annotations

import math

import torch


def attn(heads, kv_heads, dim, vdim, scale, window):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if window is not None:
        m["mask"] = dict(size=window)
    return dict(type="attention", mixer=m)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
                                                    scale=scale, rot=dict(base=base, dims=rot_dim)))


def mlstm(heads, dim, vdim, cap):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap))


def layer(mix, ff):
    return dict(type=mix["type"], mixer=dict(mix["mixer"]), mlp=None if ff is None else dict(kind="dense", ff=ff))


def config(width, vocab, eps, emb_scale, res_mult, layers, loop=None):
    """loop: (start, stop, times) or None."""
    c = dict(architecture="Zadenex", width=width, vocab=vocab, norm=dict(eps=eps), embedding=dict(scale=emb_scale),
             residual_mult=res_mult, layers=layers)
    if loop is not None:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


# A: the loop is the first three layers, three passes: a matrix memory of three heads of 16 x 24, an attention of eight heads
# over two key/value heads with keys of 20 (rows padded to 24 in the pages), values of 12 and a window of 25 (no multiple of
# anything), a latent attention whose sizes are all different.  After it a matrix memory of one head of 40 x 8 without a
# feed-forward.
CFG_A = config(64, 97, 1e-5, 1.5, 0.7, [
    layer(mlstm(3, 16, 24, 5.0), 72),
    layer(attn(8, 2, 20, 12, 0.3, 25), 40),
    layer(latent(5, 12, 8, 20, 24, 40, 0.35, 100.0), 56),
    layer(mlstm(1, 40, 8, 15.0), None),
], loop=(0, 3, 3))
# B: sizes the tensor-core kernels take; the loop is the middle layer alone, twice.  A latent attention with more rotated than
# unrotated entries, two attentions (three heads over one key/value head and a window of 70; twelve over four, no window) and
# matrix memories of 2 x (64 x 64) and 5 x (8 x 33).
CFG_B = config(96, 211, 1e-6, 4.0, 1.3, [
    layer(latent(4, 16, 32, 24, 48, 64, 0.25, 10000.0), 40),
    layer(attn(3, 1, 32, 32, 0.4, 70), 56),
    layer(mlstm(2, 64, 64, 8.0), 88),
    layer(attn(12, 4, 16, 8, 0.5, None), None),
    layer(mlstm(5, 8, 33, 2.0), 24),
], loop=(2, 3, 2))
CONFIGS = {"A": CFG_A, "B": CFG_B}
PAGE = {"A": 16, "B": 8}


def make_tensors(cfg, seed):
    """Scales that give a peaked softmax (single keys carry weight), mixing matrices far from symmetric, sinks that take a
    visible share, forget gates from nearly none to nearly all, input gates of both signs, norm weights away from 1."""
    g = torch.Generator().manual_seed(seed)
    D = cfg["width"]

    def normal(*shape, std):
        return torch.empty(shape).normal_(0.0, std, generator=g)

    def uniform(*shape, lo, hi):
        return torch.empty(shape).uniform_(lo, hi, generator=g)

    t = {"embed": normal(cfg["vocab"], D, std=0.8), "head": normal(cfg["vocab"], D, std=1.0 / math.sqrt(D)),
         "final.norm": uniform(D, lo=0.5, hi=1.5)}
    if cfg.get("loop"):
        t["loop.in"] = normal(D, 2 * D, std=1.0 / math.sqrt(2 * D))
        t["loop.step"] = normal(cfg["loop"]["times"], D, std=0.6)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        t[p + "norm1"], t[p + "norm1b"] = uniform(D, lo=0.5, hi=1.5), uniform(D, lo=0.5, hi=1.5)
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if lay["type"] == "attention":
            G = m["kv_heads"]
            t[p + "mix.q"] = normal(H * dk, D, std=1.3 / math.sqrt(D))
            t[p + "mix.k"] = normal(G * dk, D, std=1.3 / math.sqrt(D))
            t[p + "mix.v"] = normal(G * dv, D, std=1.3 / math.sqrt(D))
            for c in "qkv":
                t[f"{p}mix.{c}.b"] = normal(t[f"{p}mix.{c}"].shape[0], std=0.4)
            t[p + "mix.talk"] = normal(H, H, std=1.2 / math.sqrt(H))
            t[p + "mix.o"], t[p + "mix.o.b"] = normal(D, H * dv, std=1.0 / math.sqrt(H * dv)), normal(D, std=0.3)
        elif lay["type"] == "latent_attention":
            dr, Q, R = m["rot_dim"], m["q_rank"], m["kv_rank"]
            t[p + "mix.dq"], t[p + "mix.dq.norm"] = normal(Q, D, std=1.0 / math.sqrt(D)), uniform(Q, lo=0.5, hi=1.5)
            t[p + "mix.uq"] = normal(H * (dk + dr), Q, std=1.2 / math.sqrt(Q))
            t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = normal(R + dr, D, std=1.0 / math.sqrt(D)), uniform(R, lo=0.5, hi=1.5)
            t[p + "mix.uk"], t[p + "mix.uv"] = normal(H * dk, R, std=1.2 / math.sqrt(R)), normal(H * dv, R, std=1.0 / math.sqrt(R))
            t[p + "mix.sink"] = uniform(H, lo=-1.0, hi=3.0)
            t[p + "mix.g"], t[p + "mix.o"] = normal(H, D, std=2.0 / math.sqrt(D)), normal(D, H * dv, std=1.0 / math.sqrt(H * dv))
        else:
            for c, n in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv)):
                t[p + "mix." + c] = normal(n, D, std=1.2 / math.sqrt(D))
            # keys lean towards the queries: a head's weighted sum of values does not cancel to next to nothing, which the
            # norm behind it would magnify
            t[p + "mix.k"] = 0.6 * t[p + "mix.k"] + 0.8 * t[p + "mix.q"]
            t[p + "mix.i"], t[p + "mix.i.b"] = normal(H, D, std=1.5 / math.sqrt(D)), normal(H, std=1.0)
            t[p + "mix.f"], t[p + "mix.f.b"] = normal(H, D, std=1.5 / math.sqrt(D)), uniform(H, lo=0.0, hi=6.0)
            t[p + "mix.norm"], t[p + "mix.o"] = uniform(H * dv, lo=0.5, hi=1.5), normal(D, H * dv, std=1.0 / math.sqrt(H * dv))
        if lay.get("mlp"):
            F = lay["mlp"]["ff"]
            t[p + "norm2"], t[p + "norm2b"] = uniform(D, lo=0.5, hi=1.5), uniform(D, lo=0.5, hi=1.5)
            for c, shape in (("gate", (F, D)), ("up", (F, D)), ("down", (D, F))):
                t[f"{p}mlp.{c}"] = normal(*shape, std=1.2 / math.sqrt(shape[1]))
                t[f"{p}mlp.{c}.b"] = normal(shape[0], std=0.3)
    return {k: v.to(torch.bfloat16).float() for k, v in t.items()}

"""Small Zanelorn configurations and weights for the tests: models that differ from each other in every size and option,
with weights that make faults show."""
from __future__ import annotations

import math

import torch


def retention(heads, dim, vdim, decay, base, dims=None):
    return dict(type="retention", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay),
                                             rot=dict(base=base, dims=dim if dims is None else dims)))


def attn(heads, kv_heads, dim, vdim, scale, base, dims=None, factor=2.0, window=None, keep=0):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
             rot=dict(base=base, dims=dim if dims is None else dims, scaling=dict(factor=factor)))
    if window is not None:
        m["mask"] = dict(size=window, keep_first=keep)
    return m


def parallel(left, inner, state, dt_rank, conv, scales=(0.8, 1.1)):
    return dict(type="parallel", mixer=dict(left=left, left_scale=scales[0], right=dict(inner=inner, state=state, dt_rank=dt_rank, conv=conv),
                                            right_scale=scales[1]))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, identity, top, ff, limit, shared=None):
    """shared: (size, limit) or None."""
    m = dict(kind="moe", router=dict(experts=experts, identity=identity, top=top), expert=dict(ff=ff, limit=limit))
    if shared is not None:
        m["shared"] = dict(ff=shared[0], limit=shared[1])
    return m


def layer(mix, mlp):
    return dict(type=mix["type"], mixer=mix["mixer"], mlp=mlp)


def config(width, vocab, eps, emb_scale, res_mult, side, layers):
    return dict(architecture="Zanelorn", width=width, vocab=vocab, norm=dict(eps=eps), embedding=dict(scale=emb_scale), residual_mult=res_mult,
                token_side=dict(dim=side), layers=layers)


# A: a parallel layer whose attention has keys of 20 (rows padded to 24 in the pages) of which 8 entries turn, values of 12, a
# window of 25 and 5 kept tokens (pages of 16), and whose scan has 48 channels of 10 entries, rank 5 and 4 taps; experts with
# three identity outputs; retention heads of 16 x 24 of which all entries turn; a layer without a feed-forward.
CFG_A = config(64, 97, 1e-5, 1.5, 0.7, 12, [
    layer(parallel(attn(6, 2, 20, 12, 0.3, 100.0, dims=8, factor=3.0, window=25, keep=5), 48, 10, 5, 4), moe(7, 3, 2, 24, 1.5, (40, 2.5))),
    layer(retention(3, 16, 24, (0.9, 0.97, 0.999), 1000.0), dense(72)),
    layer(retention(1, 40, 8, (0.98,), 50.0, dims=12), None),
    layer(parallel(attn(4, 1, 16, 16, 0.4, 5e4, factor=8.0, window=60, keep=17), 40, 3, 2, 2, scales=(1.2, -0.6)), dense(40)),
])
# B: sizes the tensor-core kernels take: heads of 32 over a window of 70 with 9 kept tokens (pages of 8), no window at all,
# 96 channels of 16 entries, 24 of 40, states of 64 x 64 and 8 x 33; experts without identity outputs or without a shared one.
CFG_B = config(96, 211, 1e-6, 4.0, 0.4, 16, [
    layer(retention(2, 64, 64, (0.95, 0.998), 10000.0, dims=32), moe(12, 4, 5, 16, 3.0)),
    layer(parallel(attn(3, 3, 32, 32, 0.5, 1e4, window=70, keep=9), 96, 16, 8, 3, scales=(1.0, 1.0)), moe(5, 0, 1, 56, 0.8, (24, 4.0))),
    layer(parallel(attn(8, 4, 16, 48, 0.6, 300.0, dims=10, factor=1.5), 24, 40, 16, 5, scales=(0.5, 0.9)), dense(88)),
    layer(retention(5, 8, 33, (0.5, 0.9, 0.96, 0.99, 0.9995), 20.0, dims=6), dense(24)),
])
CONFIGS = {"A": CFG_A, "B": CFG_B}
PAGE = {"A": 16, "B": 8}


def make_tensors(cfg, seed):
    """Scales that give a peaked softmax (single keys carry weight), retention keys that lean towards the queries (the sums do
    not cancel before the norm), step sizes and rates that keep a channel's state from one token to hundreds, corrections that
    change which experts are chosen, norm weights away from 1."""
    g = torch.Generator().manual_seed(seed)
    D = cfg["width"]

    def normal(*shape, std):
        return torch.empty(shape).normal_(0.0, std, generator=g)

    def uniform(*shape, lo, hi):
        return torch.empty(shape).uniform_(lo, hi, generator=g)

    def linear(n_out, n_in, gain=1.0):
        return normal(n_out, n_in, std=gain / math.sqrt(n_in))

    unit = 1.0 / max(abs(cfg["embedding"]["scale"]), 1e-3)       # the residual starts near 1
    d = cfg["token_side"]["dim"]
    t = {"embed": normal(cfg["vocab"], D, std=unit), "head": linear(cfg["vocab"], D), "final.norm": uniform(D, lo=0.5, hi=1.5),
         "side.embed": normal(cfg["vocab"], len(cfg["layers"]) * d, std=1.0)}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        t[p + "norm1"] = uniform(D, lo=0.5, hi=1.5)
        if lay["type"] == "retention":
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            for c, n in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv)):
                t[p + "mix." + c] = linear(n, D, 1.2)
            t[p + "mix.k"] = 0.6 * t[p + "mix.k"] + 0.8 * t[p + "mix.q"]
            t[p + "mix.o"] = linear(D, H * dv)
        else:
            a, r = m["left"], m["right"]
            q = p + "mix.left."
            for c, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                t[q + c], t[q + c + ".b"] = linear(n, D, 1.3), normal(n, std=0.4)
            t[q + "q.norm"], t[q + "k.norm"] = uniform(a["dim"], lo=0.8, hi=1.8), uniform(a["dim"], lo=0.8, hi=1.8)
            t[q + "g"], t[q + "o"] = linear(a["heads"] * a["vdim"], D, 1.5), linear(D, a["heads"] * a["vdim"])
            I, N, R, K = r["inner"], r["state"], r["dt_rank"], r["conv"]
            q = p + "mix.right."
            t[q + "in"], t[q + "conv"], t[q + "conv.b"] = linear(2 * I, D, 1.3), linear(I, K, 1.2), normal(I, std=0.2)
            t[q + "x"], t[q + "dt"], t[q + "dt.b"] = linear(R + 2 * N, I, 1.2), linear(I, R, 1.0), uniform(I, lo=-4.0, hi=0.5)
            t[q + "A_log"], t[q + "D"], t[q + "o"] = uniform(I, N, lo=-3.0, hi=1.5), uniform(I, lo=-1.0, hi=1.0), linear(D, I)
        f = lay.get("mlp")
        if f:
            t[p + "norm2"] = uniform(D, lo=0.5, hi=1.5)
            if f["kind"] == "dense":
                t[p + "mlp.up"], t[p + "mlp.down"] = linear(f["ff"], D, 1.3), linear(D, f["ff"], 1.3)
            else:
                E, n = f["router"]["experts"], f["router"]["experts"] + f["router"]["identity"]
                t[p + "mlp.router"], t[p + "mlp.correction"] = linear(n, D, 2.0), normal(n, std=0.1)
                for e in range(E):
                    for c, shape in (("gate", (f["expert"]["ff"], D)), ("up", (f["expert"]["ff"], D)), ("down", (D, f["expert"]["ff"]))):
                        t[f"{p}mlp.e{e}.{c}"] = linear(*shape, 1.5)
                if f.get("shared"):
                    for c, shape in (("gate", (f["shared"]["ff"], D)), ("up", (f["shared"]["ff"], D)), ("down", (D, f["shared"]["ff"]))):
                        t[f"{p}mlp.shared.{c}"] = linear(*shape, 1.5)
                    t[p + "mlp.shared.sg"] = linear(1, D, 1.5)
        t[p + "side.gate"], t[p + "side.proj"], t[p + "side.norm"] = linear(d, D, 1.3), linear(D, d), uniform(D, lo=0.5, hi=1.5)
    return {k: v.to(torch.bfloat16).float() for k, v in t.items()}

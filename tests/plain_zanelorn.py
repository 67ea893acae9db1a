"""A plain, slow statement of the Zanelorn design: whole sequences, no cache, float64.

One function per mechanism, written from the design's equations; it shares no code with
the package.  ``tensors`` maps checkpoint names to torch tensors, ``cfg`` is the parsed
config.json.  ``store`` rounds the values that the engine hands from kernel to kernel in
its activation dtype (identity for the 32-bit path).

Notation: D width, T tokens, p position (from 0).  Retention: Hr heads with a state S [dk, dv] and
a decay each.  Attention: H query heads over G key/value heads, w the window, f the first tokens that stay
visible.  Selective scan: C channels with a state of N entries each.
"""
from __future__ import annotations

import math
from typing import Callable, Dict, List, Optional, Sequence

import torch

F64 = torch.float64
SIGMOID_FACTOR = 1.702


def _keep(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(F64)


def rms_unit(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------------------- rotation
def rotate_halves(x, positions, dims: int, base: float, factor: float = 1.0):
    """x [..., T, d]: entries i and i + dims/2 of the first ``dims``, read as one complex number, are multiplied by e^(j a),
    a = position * base^(-2i/dims) / factor.  The angle is taken in 32-bit: frequency and position as float32, their product
    rounded to float32."""
    if dims == 0:
        return x
    half = dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=F64) / dims) / factor
    a = (positions.to(torch.float32)[:, None] * f.to(torch.float32)[None, :]).to(F64)
    cos, sin = torch.cos(a), torch.sin(a)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


# ------------------------------------------------------------------------------------------- retention
def retention_scan(q, k, v, decay: Sequence[float], state=None):
    """Head by head, from S = 0: S <- a_h S + k v^T (a_h: ``decay``), o = S^T q.  q, k [T, Hr, dk], v [T, Hr, dv]; returns
    (o [T, Hr, dv], S)."""
    T, Hr, dk = q.shape
    dv = v.shape[2]
    S = torch.zeros(Hr, dk, dv, dtype=F64) if state is None else state.clone()
    a = torch.tensor(decay, dtype=F64)[:, None, None]
    out = torch.zeros(T, Hr, dv, dtype=F64)
    for t in range(T):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    return out, S


def retention(h, w: Dict[str, torch.Tensor], m: dict, eps: float, store: Callable = _keep):
    """h [T, D] -> [T, D]."""
    T, Hr, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)

    def heads(c):
        x = (h @ w[c].T).view(T, Hr, dk).transpose(0, 1)
        return rotate_halves(x, pos, m["rot"]["dims"], m["rot"]["base"]).transpose(0, 1)

    q, k = heads("q"), heads("k") * dk ** -0.5
    o, _ = retention_scan(q, k, (h @ w["v"].T).view(T, Hr, dv), m["decay"])
    y = rms_unit(o, eps).reshape(T, Hr * dv) * silu(h @ w["g"].T)
    return store(y) @ w["o"].T


# ------------------------------------------------------------------------------------------- softmax attention
def visible(T: int, window: Optional[int], keep_first: int = 0):
    """mask[i, j]: query i sees key j: j <= i and (i - j < window or j < keep_first)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    m = j <= i
    if window:
        m = m & ((i - j < window) | (j < keep_first))
    return m


def softmax_attention(q, k, v, scale: float, mask):
    """q [H, T, dk], k [G, T, dk], v [G, T, dv] -> [H, T, dv]: query head h reads key/value head floor(h / (H / G))."""
    R = q.shape[0] // k.shape[0]
    k, v = k.repeat_interleave(R, 0), v.repeat_interleave(R, 0)
    s = (q @ k.transpose(1, 2)) * scale
    return torch.softmax(s.masked_fill(~mask[None], float("-inf")), -1) @ v


def gated_attention(h, w: Dict[str, torch.Tensor], m: dict, eps: float, store: Callable = _keep):
    """h [T, D] -> the joined heads [T, H * dv] times sigmoid(W_g h), before the output projection."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot, pos = m["rot"], torch.arange(h.shape[0])
    factor = (rot.get("scaling") or {}).get("factor", 1.0)

    def heads(c, n, d):
        return store(h @ w[c].T + w[c + ".b"]).view(T, n, d).transpose(0, 1)

    def turned(c, n):
        return store(rotate_halves(rms_norm(heads(c, n, dk), w[c + ".norm"], eps), pos, rot["dims"], rot["base"], factor))

    mask = m.get("mask") or {}
    o = softmax_attention(turned("q", H), turned("k", G), heads("v", G, dv), m["scale"],
                          visible(T, mask.get("size"), mask.get("keep_first") or 0))
    return o.transpose(0, 1).reshape(T, H * dv) * torch.sigmoid(store(h @ w["g"].T))


# ------------------------------------------------------------------------------------------- selective scan
def causal_conv(x, weight, bias):
    """x [T, C] -> [T, C]: y_t = b + sum_j weight[:, j] x_(t - taps + 1 + j), zeros before the start."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F64), x])
    return bias + sum(padded[j:j + x.shape[0]] * weight[:, j] for j in range(taps))


def selective_scan(x, dt, A, B, C, skip, state=None):
    """Every channel's row s of S: s <- e^(dt a) * s + dt x B (a its row of A), y = s . C + skip x.  x, dt [T, channels],
    A [channels, N], B, C [T, N]; returns (y [T, channels], S)."""
    S = torch.zeros_like(A) if state is None else state.clone()
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + skip * x[t]
    return y, S


def mamba(h, w: Dict[str, torch.Tensor], m: dict, store: Callable = _keep):
    """h [T, D] -> [T, inner], before the output projection."""
    inner, N, R = m["inner"], m["state"], m["dt_rank"]
    xz = store(h @ w["in"].T)
    x = store(silu(causal_conv(xz[:, :inner], w["conv"], w["conv.b"])))
    low = store(x @ w["x"].T)
    dt = softplus(low[:, :R] @ w["dt"].T + w["dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(w["A_log"]), low[:, R:R + N], low[:, R + N:], w["D"])
    return y * silu(xz[:, inner:])


def parallel(h, w: Dict[str, torch.Tensor], m: dict, eps: float, store: Callable = _keep):
    """Both branches read h; their results are added with the two constants."""
    left, right = sub(w, "left."), sub(w, "right.")
    a = store(gated_attention(h, left, m["left"], eps, store) * m["left_scale"]) @ left["o"].T
    b = store(mamba(h, right, m["right"], store) * m["right_scale"]) @ right["o"].T
    return a + b


# ------------------------------------------------------------------------------------------- feed-forward
def dense_ff(h, w: Dict[str, torch.Tensor], store: Callable = _keep):
    return store(gelu_erf(h @ w["up"].T)) @ w["down"].T


def clamped_expert(h, gate, up, down, limit: float, store: Callable = _keep):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return store(g * torch.sigmoid(SIGMOID_FACTOR * g) * (u + 1.0)) @ down.T


def choose(z, correction, top: int):
    """z [T, E] -> (experts [T, top], weights [T, top]): scores s = softmax(z); the largest s + correction are chosen and
    weighted by s as it is."""
    s = torch.softmax(z, -1)
    idx = torch.topk(s + correction, top, -1).indices
    return idx, torch.gather(s, -1, idx)


def moe(h, w: Dict[str, torch.Tensor], m: dict, store: Callable = _keep):
    E = m["router"]["experts"]
    idx, wt = choose(h @ w["router"].T, w["correction"], m["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(idx[t].tolist(), wt[t]):
            if e < E:
                y[t] += a * clamped_expert(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], m["expert"]["limit"], store)[0]
            else:                       # an expert that gives its input back
                y[t] += a * h[t]
    if m.get("shared"):
        y = y + torch.sigmoid(h @ w["shared.sg"].T) * clamped_expert(h, w["shared.gate"], w["shared.up"], w["shared.down"],
                                                                     m["shared"]["limit"], store)
    return y


# ------------------------------------------------------------------------------------------- the model
def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def token_side(h, row, w: Dict[str, torch.Tensor], eps: float, store: Callable = _keep):
    """h [T, D], row [T, d] (the layer's part of the tokens' rows in the side table) -> [T, D]."""
    return rms_norm(store(gelu_tanh(h @ w["gate"].T) * row) @ w["proj"].T, w["norm"], eps)


def layer(x, ids, tensors, cfg, i: int, store: Callable = _keep):
    eps, m, lay, p = cfg["norm"]["eps"], float(cfg["residual_mult"]), cfg["layers"][i], f"l{i}."
    mw = sub(tensors, p + "mix.")
    h = store(x)
    y = retention(h, mw, lay["mixer"], eps, store) if lay["type"] == "retention" else parallel(h, mw, lay["mixer"], eps, store)
    x = x + m * rms_norm(y, tensors[p + "norm1"].to(F64), eps)
    if lay.get("mlp"):
        ff = dense_ff(store(x), sub(tensors, p + "mlp."), store) if lay["mlp"]["kind"] == "dense" \
            else moe(store(x), sub(tensors, p + "mlp."), lay["mlp"], store)
        x = x + m * rms_norm(ff, tensors[p + "norm2"].to(F64), eps)
    d = cfg["token_side"]["dim"]
    row = tensors["side.embed"].to(F64)[ids][:, i * d:(i + 1) * d]
    return x + m * token_side(store(x), row, sub(tensors, p + "side."), eps, store)


def forward(tensors: Dict[str, torch.Tensor], cfg: dict, tokens, store: Callable = _keep, trace: Optional[list] = None):
    """Logits [T, vocab] of a whole sequence.  ``trace``: gets the residual after every layer."""
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = tensors["embed"].to(F64)[ids] * float(cfg["embedding"]["scale"])
    for i in range(len(cfg["layers"])):
        x = layer(x, ids, tensors, cfg, i, store)
        if trace is not None:
            trace.append(x.clone())
    y = rms_norm(x, tensors["final.norm"].to(F64), cfg["norm"]["eps"])
    return store(y) @ tensors["head"].to(F64).T


def greedy(tensors, cfg, prompt, n_new: int, store: Callable = _keep) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(tensors, cfg, toks, store)[-1])))
    return toks[len(prompt):]

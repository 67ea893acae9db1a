"""A plain, slow statement of the Zadenex design: whole sequences, no cache, float64.

One function per mechanism, written from the design's equations; it shares no code with
the package.  ``tensors`` maps checkpoint names to torch tensors, ``cfg`` is the parsed
config.json.  ``store`` rounds the values that the engine hands from kernel to kernel in
its activation dtype (identity for the 32-bit path); ``tables`` likewise the rows of the embedding.

Notation: D width, T tokens, p position (from 0).  Attention: H query heads over G key/value
heads, dk query/key size, dv value size, w the window.  Latent attention: R the latent's size, dn
unrotated and dr rotated columns per head.  Matrix memory: Hm heads with a state S [dk, dv], a row
sum n [dk] and a running maximum m per head.
"""
from __future__ import annotations

import math
from typing import Callable, Dict, List, Optional

import torch

F64 = torch.float64


def _keep(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(F64)


def rms_unit(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------- softmax attention
def visible(T: int, window: Optional[int]):
    """mask[i, j]: query i sees key j: j <= i and (with a window) i - j < window."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    m = j <= i
    if window:
        m = m & (i - j < window)
    return m


def mix_heads(s, talk):
    """Scores of head h: sum_g talk[h, g] * s_g.  s [H, T, T], talk [H, H]."""
    return torch.einsum("hg,gij->hij", talk, s)


def softmax_with_sink(s, sink):
    """exp(s_j) / (exp(sink_h) + sum_j exp(s_j)) over the last axis; s [H, T, T] with -inf where nothing is seen."""
    sink = sink.to(F64)[:, None, None]
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (torch.exp(sink - top) + e.sum(-1, keepdim=True))


def attention(h, w: Dict[str, torch.Tensor], m: dict, store: Callable = _keep):
    """h [T, D] -> [T, D]: biases on all four projections, scores mixed over the heads, a window, a sink of score 0."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = store(h @ w["q"].T + w["q.b"]).view(T, H, dk).transpose(0, 1)
    k = store(h @ w["k"].T + w["k.b"]).view(T, G, dk).transpose(0, 1)
    v = store(h @ w["v"].T + w["v.b"]).view(T, G, dv).transpose(0, 1)
    k = k.repeat_interleave(H // G, 0)
    v = v.repeat_interleave(H // G, 0)
    s = mix_heads((q @ k.transpose(1, 2)) * m["scale"], w["talk"])
    s = s.masked_fill(~visible(T, (m.get("mask") or {}).get("size"))[None], float("-inf"))
    p = softmax_with_sink(s, torch.zeros(H, dtype=F64))
    o = store((p @ v).transpose(0, 1).reshape(T, H * dv))
    return o @ w["o"].T + w["o.b"]


# ------------------------------------------------------------------------------------------- latent attention
def rotate_pairs(x, positions, dims: int, base: float):
    """x [..., T, d]: entries 2i and 2i + 1 of the first ``dims`` are a pair (u, v); at position p it becomes
    (u cos a - v sin a, v cos a + u sin a), a = p * base^(-2i/dims).  The angle is taken in 32-bit: frequency and position
    as float32, their product rounded to float32."""
    if dims == 0:
        return x
    i = torch.arange(dims // 2, dtype=F64)
    f = float(base) ** (-2.0 * i / dims)
    a = (positions.to(torch.float32)[:, None] * f.to(torch.float32)[None, :]).to(F64)
    cos, sin = torch.cos(a), torch.sin(a)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def latent_queries(h, w, m: dict, eps: float, store: Callable = _keep):
    """(unrotated [H, T, dn], rotated [H, T, dr]) through the queries' latent."""
    T, H, dn, dr = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    cq = store(rms_norm(store(h @ w["dq"].T), w["dq.norm"], eps))
    q = store(cq @ w["uq"].T).view(T, H, dn + dr).transpose(0, 1)
    return q[..., :dn], rotate_pairs(q[..., dn:], torch.arange(T), m["rot"]["dims"], m["rot"]["base"])


def latent_rows(h, w, m: dict, eps: float, store: Callable = _keep):
    """What is cached of every token: (the latent [T, R], the shared rotated key part [T, dr])."""
    R = m["kv_rank"]
    d = store(h @ w["dkv"].T)
    c = store(rms_norm(d[:, :R], w["dkv.norm"], eps))
    return c, store(rotate_pairs(d[:, R:], torch.arange(h.shape[0]), m["rot"]["dims"], m["rot"]["base"]))


def latent_attention(h, w: Dict[str, torch.Tensor], m: dict, eps: float, store: Callable = _keep):
    """h [T, D] -> [T, D]."""
    T = h.shape[0]
    H, dn, dv = m["heads"], m["dim"], m["vdim"]
    qn, qr = latent_queries(h, w, m, eps, store)
    c, kr = latent_rows(h, w, m, eps, store)
    kn = (c @ w["uk"].T).view(T, H, dn).transpose(0, 1)
    v = (c @ w["uv"].T).view(T, H, dv).transpose(0, 1)
    s = (qn @ kn.transpose(1, 2) + qr @ kr.T[None]) * m["scale"]
    s = s.masked_fill(~visible(T, None)[None], float("-inf"))
    o = softmax_with_sink(s, w["sink"]) @ v
    gate = torch.sigmoid(store(h @ w["g"].T))
    o = store((o * gate.T[:, :, None]).transpose(0, 1).reshape(T, H * dv))
    return o @ w["o"].T


# ------------------------------------------------------------------------------------------- matrix memory
def memory_gates(h, w, m: dict):
    """(i, f) [T, Hm]: the log input gate cap * tanh((W_i h + b) / cap) and the log forget gate
    logsigmoid(cap * tanh((W_f h + b) / cap))."""
    cap = m["gate_cap"]
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap))
    return i, f


def memory_scan(q, k, v, i, f, state=None):
    """Per head, with S, n and m zero at the start: m' = max(f + m, i); S = exp(f + m - m') S + exp(i - m') k v^T;
    n likewise with k alone; o = S^T q / (max(|n . q|, exp(-m')) + 1e-6).  q, k [T, Hm, dk], v [T, Hm, dv], i, f [T, Hm];
    returns (o [T, Hm, dv], (S, n, m))."""
    T, Hm, dk = q.shape
    dv = v.shape[2]
    if state is None:
        S, n, mx = torch.zeros(Hm, dk, dv, dtype=F64), torch.zeros(Hm, dk, dtype=F64), torch.zeros(Hm, dtype=F64)
    else:
        S, n, mx = (t.clone() for t in state)
    out = torch.zeros(T, Hm, dv, dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + mx, i[t])
        a, b = torch.exp(f[t] + mx - new), torch.exp(i[t] - new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        mx = new
        num = torch.einsum("hij,hi->hj", S, q[t])
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-mx)) + 1e-6
        out[t] = num / den[:, None]
    return out, (S, n, mx)


def mlstm(h, w: Dict[str, torch.Tensor], m: dict, eps: float, store: Callable = _keep):
    """h [T, D] -> [T, D]."""
    T = h.shape[0]
    Hm, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, Hm, dk) * dk ** -0.5
    k = (h @ w["k"].T).view(T, Hm, dk)
    v = (h @ w["v"].T).view(T, Hm, dv)
    i, f = memory_gates(h, w, m)
    o, _ = memory_scan(q, k, v, i, f)
    y = rms_unit(o, eps).reshape(T, Hm * dv) * w["norm"] * torch.sigmoid(h @ w["g"].T)
    return store(y) @ w["o"].T


# ------------------------------------------------------------------------------------------- feed-forward
def dense_ff(h, w: Dict[str, torch.Tensor], store: Callable = _keep):
    """W_down (gelu_tanh(W_gate h) * (W_up h)), biases on all three."""
    g, u = store(h @ w["gate"].T + w["gate.b"]), store(h @ w["up"].T + w["up.b"])
    return store(gelu_tanh(g) * u) @ w["down"].T + w["down.b"]


# ------------------------------------------------------------------------------------------- the model
def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def layer_runs(cfg: dict):
    """[(layer, number of the pass that begins right before it, or None)] in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def enter_pass(x, x0, w_in, step):
    """x <- W_in [x; x0] + the pass's vector."""
    return torch.cat([x, x0], -1) @ w_in.T + step


def layer(x, tensors, cfg, i: int, store: Callable = _keep):
    eps, m, lay, p = cfg["norm"]["eps"], float(cfg["residual_mult"]), cfg["layers"][i], f"l{i}."
    norm = {k: tensors[p + k].to(F64) for k in ("norm1", "norm1b", "norm2", "norm2b") if p + k in tensors}
    mw = sub(tensors, p + "mix.")
    h = store(rms_norm(x, norm["norm1"], eps))
    if lay["type"] == "mlstm":
        y = mlstm(h, mw, lay["mixer"], eps, store)
    elif lay["type"] == "latent_attention":
        y = latent_attention(h, mw, lay["mixer"], eps, store)
    else:
        y = attention(h, mw, lay["mixer"], store)
    x = x + m * rms_norm(y, norm["norm1b"], eps)
    if lay.get("mlp"):
        h = store(rms_norm(x, norm["norm2"], eps))
        x = x + m * rms_norm(dense_ff(h, sub(tensors, p + "mlp."), store), norm["norm2b"], eps)
    return x


def forward(tensors: Dict[str, torch.Tensor], cfg: dict, tokens, store: Callable = _keep, trace: Optional[list] = None):
    """Logits [T, vocab] of a whole sequence.  ``trace``: gets the residual after every layer run."""
    E = tensors["embed"].to(F64)
    x0 = E[torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    x = x0
    for i, t in layer_runs(cfg):
        if t is not None:
            x = enter_pass(x, x0, tensors["loop.in"].to(F64), tensors["loop.step"][t].to(F64))
        x = layer(x, tensors, cfg, i, store)
        if trace is not None:
            trace.append(x.clone())
    y = rms_norm(x, tensors["final.norm"].to(F64), cfg["norm"]["eps"])
    return store(y) @ tensors["head"].to(F64).T


def greedy(tensors, cfg, prompt, n_new: int, store: Callable = _keep) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(tensors, cfg, toks, store)[-1])))
    return toks[len(prompt):]

"""A recurrent mixer with a matrix memory and exponential gates (the mLSTM cell of xLSTM).

q_t = W_q h / sqrt(dim), k_t = W_k h (heads of ``head_dim``), v_t = W_v h (heads of ``v_head_dim``).  Per head a log input
gate i_t = c tanh((W_i h + b_i) / c) and a log forget gate f_t = logsigmoid(c tanh((W_f h + b_f) / c)), c = ``gate_cap``.
With a state S [dim, vdim], n [dim] and a running maximum m, all zero at the start of a sequence:

    m_t = max(f_t + m_(t-1), i_t)      a = exp(f_t + m_(t-1) - m_t)      b = exp(i_t - m_t)
    S_t = a S_(t-1) + b k_t v_t^T      n_t = a n_(t-1) + b k_t
    o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + denom_eps)

Each head's o_t is divided by its root mean square (eps inside the root); the joined heads are multiplied by a weight per
channel and by sigmoid(W_g h), then W_o.  The six input matrices are one product whose result stays 32-bit (its columns enter
the recurrence); the gates, the state, o, the norm and the output gate are 32-bit whatever the engine's dtype.  The request's
state is S, n and m of every head in one row of the cache manager's state arena.
"""
from __future__ import annotations

from ..cache.manager import StateNeed
from .base import ParamSpec, register_part
from .projected import ProjectedMixer


class MatrixMemoryMixer(ProjectedMixer):
    in_names = ("q_weight", "k_weight", "v_weight", "g_weight", "i_weight", "f_weight")
    out_name = "out_weight"
    proj_f32 = True

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int, gate_cap: float, norm_eps: float,
                 denom_eps: float = 1e-6):
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        self.gate_cap, self.norm_eps, self.denom_eps = float(gate_cap), float(norm_eps), float(denom_eps)
        if not self.gate_cap > 0:
            raise ValueError(f"matrix memory: the cap on the gates must be positive, got {gate_cap!r}")
        H = self.num_heads
        nk, nv = H * self.head_dim, H * self.v_head_dim
        self.cols = {"q": 0, "k": nk, "v": 2 * nk, "g": 2 * nk + nv, "i": 2 * nk + 2 * nv, "f": 2 * nk + 2 * nv + H}
        self.inner = nv
        self.state_floats = H * (self.head_dim * (self.v_head_dim + 1) + 1)

    def param_specs(self):
        D, H = self.hidden_size, self.num_heads
        nk = H * self.head_dim
        return {"q_weight": ParamSpec((nk, D), "matrix"), "k_weight": ParamSpec((nk, D), "matrix"),
                "v_weight": ParamSpec((self.inner, D), "matrix"), "g_weight": ParamSpec((self.inner, D), "matrix"),
                "i_weight": ParamSpec((H, D), "matrix"), "i_bias": ParamSpec((H,), "vector"),
                "f_weight": ParamSpec((H, D), "matrix"), "f_bias": ParamSpec((H,), "vector"),
                "norm_weight": ParamSpec((self.inner,), "vector"), "out_weight": ParamSpec((D, self.inner), "matrix")}

    def kernel_limits(self, dtype: str):
        from .. import ops
        if max(self.head_dim, self.v_head_dim) > ops.MLSTM_MAX_DIM:
            return [f"matrix memory: states of {self.head_dim} x {self.v_head_dim} per head; the kernels take up to "
                    f"{ops.MLSTM_MAX_DIM} x {ops.MLSTM_MAX_DIM}"]
        return []

    def cache_need(self):
        return StateNeed((self.state_floats,), "float32")

    def bind(self, params, rt) -> None:
        import torch
        super().bind(params, rt)
        if "i_bias" in params:      # the gates' biases ride in the input product
            self.in_bias = torch.zeros(self.in_width, dtype=torch.float32, device=self.i_bias.device)
            self.in_bias[self.cols["i"]:self.cols["f"]] = self.i_bias
            self.in_bias[self.cols["f"]:] = self.f_bias

    def core(self, proj, ctx, cache, out, out_scale: float = 1.0) -> None:
        import torch
        if out_scale != 1.0:
            raise NotImplementedError("matrix memory takes no branch factor")
        ops = self.rt.ops
        T, H = proj.shape[0], self.num_heads
        sizes = dict(heads=H, dim=self.head_dim, vdim=self.v_head_dim, write_state=cache.write)
        norms = dict(q_scale=self.head_dim ** -0.5, denom_eps=self.denom_eps, eps=self.norm_eps)
        if getattr(ctx, "decode_only", False) and ops.mlstm_step_ok(self.head_dim, self.v_head_dim):
            ops.mlstm_step(proj, self.cols, self.norm_weight, cache.state, ctx, out, cap=self.gate_cap, **norms, **sizes)
            return
        raw = ctx.ws.buf("mlstm_raw", T, self.inner, torch.float32)
        aux = ctx.ws.buf("mlstm_aux", T, 2 * H, torch.float32)
        ops.mlstm_scan(proj, self.cols, cache.state, ctx, raw, aux, cap=self.gate_cap, **sizes)
        ops.mlstm_finish(raw, aux, proj, self.cols, self.norm_weight, cache.state, ctx, out, **norms, **sizes)


register_part("mixer", "matrix_memory", MatrixMemoryMixer)

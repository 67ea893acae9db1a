"""Retention (RetNet): a matrix memory per head that forgets at a constant rate.

Queries and keys (heads of ``head_dim`` entries, bias-free projections) are turned by their position (``rot_dims`` entries,
``parts.rotary``) and the turned keys scaled by head_dim^(-1/2); values are heads of ``v_head_dim``.  A head with the constant
a keeps S [dim, vdim], at first all zeros:

    S <- a S + k v^T        o = S^T q

o is brought to unit root mean square (eps inside the root) head by head, gated with silu of a fourth projection, and
projected by W_o.  The four input matrices are one product whose result stays 32-bit (its columns enter the recurrence);
the rotation, the state, o, the norm and the gate are 32-bit whatever the engine's dtype.  The request's state is S of every
head in one row of the cache manager's state arena.
"""
from __future__ import annotations

from typing import Optional, Sequence

from ..cache.manager import StateNeed
from .base import ParamSpec, register_part
from .projected import ProjectedMixer
from .rotary import rotary_table


class RetentionMixer(ProjectedMixer):
    in_names = ("q_weight", "k_weight", "v_weight", "g_weight")
    out_name = "out_weight"
    proj_f32 = True

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int, decay: Sequence[float], norm_eps: float,
                 rot_dims: int = 0, rot_base: float = 10000.0, rot_interleaved: bool = False, rot_scaling: Optional[dict] = None):
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        self.decay_values = [float(a) for a in decay]
        if len(self.decay_values) != self.num_heads:
            raise ValueError(f"retention: {len(self.decay_values)} decays for {num_heads} heads")
        self.norm_eps = float(norm_eps)
        self.rot_dims, self.rot_base, self.rot_interleaved = int(rot_dims), float(rot_base), bool(rot_interleaved)
        self.rot_scaling = None if rot_scaling is None else dict(rot_scaling)
        if self.rot_dims < 0 or self.rot_dims % 2 or self.rot_dims > self.head_dim:
            raise ValueError(f"rot_dims={rot_dims} must be even and at most head_dim={head_dim}")
        nk, nv = self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        self.cols = {"q": 0, "k": nk, "v": 2 * nk, "g": 2 * nk + nv}
        self.inner = nv
        self.state_floats = nk * self.v_head_dim
        self.freq = self.decay = None

    def param_specs(self):
        D, nk = self.hidden_size, self.num_heads * self.head_dim
        return {"q_weight": ParamSpec((nk, D), "matrix"), "k_weight": ParamSpec((nk, D), "matrix"),
                "v_weight": ParamSpec((self.inner, D), "matrix"), "g_weight": ParamSpec((self.inner, D), "matrix"),
                "out_weight": ParamSpec((D, self.inner), "matrix")}

    def kernel_limits(self, dtype: str):
        from .. import ops
        if max(self.head_dim, self.v_head_dim) > ops.RETENTION_MAX_DIM:
            return [f"retention: states of {self.head_dim} x {self.v_head_dim} per head; the kernels take up to "
                    f"{ops.RETENTION_MAX_DIM} x {ops.RETENTION_MAX_DIM}"]
        return []

    def cache_need(self):
        return StateNeed((self.state_floats,), "float32")

    def bind(self, params, rt) -> None:
        import torch
        super().bind(params, rt)
        self.decay = torch.tensor(self.decay_values, dtype=torch.float64).float().to(rt.device)
        if self.rot_dims:
            f, _ = rotary_table(self.rot_dims, self.rot_base, self.rot_scaling)
            self.freq = torch.tensor(f, dtype=torch.float64).float().contiguous().to(rt.device)

    def core(self, proj, ctx, cache, out, out_scale: float = 1.0) -> None:
        import torch
        if out_scale != 1.0:
            raise NotImplementedError("retention takes no branch factor")
        ops = self.rt.ops
        T = proj.shape[0]
        sizes = dict(heads=self.num_heads, dim=self.head_dim, vdim=self.v_head_dim)
        rot = dict(freq=self.freq, rot_dims=self.rot_dims, interleaved=self.rot_interleaved, k_scale=self.head_dim ** -0.5)
        if getattr(ctx, "decode_only", False) and ops.retention_step_ok(self.head_dim, self.v_head_dim):
            ops.retention_step(proj, self.cols, self.decay, cache.state, ctx, out, eps=self.norm_eps, write_state=cache.write, **rot, **sizes)
            return
        ops.rotate_heads(proj, self.cols["q"], self.cols["k"], ctx, heads=self.num_heads, dim=self.head_dim, **rot)
        raw = ctx.ws.buf("retention_raw", T, self.inner, torch.float32)
        ops.retention_scan(proj, self.cols, self.decay, cache.state, ctx, raw, write_state=cache.write, **sizes)
        ops.retention_finish(raw, proj, self.cols["g"], out, heads=self.num_heads, vdim=self.v_head_dim, eps=self.norm_eps)


register_part("mixer", "retention", RetentionMixer)

"""State-space mixers: a fixed-size state per request, carried from token to token (``MambaMixer``: see the class).

``Mamba2Mixer`` (state-space duality).  With inner = heads * vdim, N state rows and G groups, W_in h is
[z: inner | x: inner | B: G*N | C: G*N | dt: heads].  x, B and C pass a causal convolution per channel (weights
[channels, taps], the last column the current token's, zeros before the start of a sequence, a bias) and silu.
dt <- softplus(dt + dt_bias).  Per head h (group floor(h / (heads / G))), with a state S [N, vdim] that starts at zero:

    S_t = exp(-exp(A_log_h) dt_t) S_(t-1) + dt_t B_t x_t^T        y_t = S_t^T C_t + D_h x_t

The joined y is multiplied by silu(z), RMS-normed in ``norm_groups`` equal parts (each by its own root mean square),
multiplied by a weight, and projected by W_o.  The request's state holds S of every head and the last taps - 1 inputs
of the convolution, both 32-bit, in one row of the cache manager's state arena; dt, the decay and the recurrence are
32-bit whatever the engine's dtype.
"""
from __future__ import annotations

from ..cache.manager import StateNeed
from .base import ParamSpec, register_part
from .projected import ProjectedMixer


class Mamba2Mixer(ProjectedMixer):
    in_names = ("in_proj",)
    out_name = "out_weight"

    def __init__(self, hidden_size: int, num_heads: int, v_head_dim: int, state_size: int, groups: int, conv_taps: int,
                 norm_groups: int, norm_eps: float):
        self.hidden_size, self.num_heads, self.v_head_dim = int(hidden_size), int(num_heads), int(v_head_dim)
        self.state_size, self.groups, self.conv_taps = int(state_size), int(groups), int(conv_taps)
        self.norm_groups, self.norm_eps = int(norm_groups), float(norm_eps)
        self.inner = self.num_heads * self.v_head_dim
        self.channels = self.inner + 2 * self.groups * self.state_size
        if self.num_heads % self.groups:
            raise ValueError(f"mamba2: {self.num_heads} heads in {self.groups} groups")
        if self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.inner} columns in {self.norm_groups} norm groups")
        self.ssm_floats = self.num_heads * self.state_size * self.v_head_dim
        self.state_floats = self.ssm_floats + (self.conv_taps - 1) * self.channels

    def param_specs(self):
        Hm = self.num_heads
        return {"in_proj": ParamSpec((2 * self.inner + 2 * self.groups * self.state_size + Hm, self.hidden_size), "matrix"),
                "conv_weight": ParamSpec((self.channels, self.conv_taps), "vector"),
                "conv_bias": ParamSpec((self.channels,), "vector"),
                "dt_bias": ParamSpec((Hm,), "vector"),
                "A_log": ParamSpec((Hm,), "vector"),
                "D": ParamSpec((Hm,), "vector"),
                "norm_weight": ParamSpec((self.inner,), "vector"),
                "out_weight": ParamSpec((self.hidden_size, self.inner), "matrix")}

    def kernel_limits(self, dtype: str):
        from .. import ops
        out = []
        if self.state_size > ops.SSD_MAX_STATE_ROWS:
            out.append(f"mamba2: a state of {self.state_size} rows per head; the kernel takes {ops.SSD_MAX_STATE_ROWS}")
        if not (1 <= self.conv_taps <= ops.SSD_MAX_TAPS):
            out.append(f"mamba2: a convolution of {self.conv_taps} taps; the kernel takes 1 to {ops.SSD_MAX_TAPS}")
        return out

    def cache_need(self):
        return StateNeed((self.state_floats,), "float32")

    def core(self, proj, ctx, cache, out, out_scale: float = 1.0) -> None:
        import torch
        if out_scale != 1.0:
            raise NotImplementedError("mamba2 takes no branch factor")
        ops = self.rt.ops
        T = proj.shape[0]
        xbc = ctx.ws.buf("ssd_xbc", T, self.channels, torch.float32)
        ops.ssd_conv(proj, self.inner, self.conv_weight, self.conv_bias, cache.state, self.ssm_floats, ctx, xbc,
                     write_state=cache.write)
        y = ctx.ws.buf("ssd_y", T, self.inner, torch.float32)
        ops.ssd_scan(xbc, proj, self.inner + self.channels, self.dt_bias, self.A_log, self.D, cache.state, ctx, y,
                     heads=self.num_heads, vdim=self.v_head_dim, state_rows=self.state_size, groups=self.groups,
                     write_state=cache.write)
        ops.gated_group_norm(y, proj[:, :self.inner], self.norm_weight, out, self.norm_groups, self.norm_eps)


register_part("mixer", "mamba2", Mamba2Mixer)


class MambaMixer(ProjectedMixer):
    """The selective scan with a state vector per channel (Mamba's first form).  One product gives ``inner`` inputs and as many
    gates z; the inputs go through Mamba-2's short convolution (with bias and silu) to x; a second product of x gives, side by
    side, a low-rank step size of ``dt_rank`` numbers and the vectors B and C of ``state_size`` entries; a third one spreads the
    step size over the channels, h = softplus(W_dt low + bias).  Channel c with the rates a = -exp(A_log[c]) keeps s, at first
    zeros:

        s <- e^(h a) * s + h x B   (entry by entry)        y = s . C + D_c x

    and the mixer's result is W_o (y * silu(z)).  The request's state holds the channels' s and the last taps - 1 inputs of the convolution, both 32-bit, in one
    row of the cache manager's state arena; dt, the decays, the recurrence and the gate are 32-bit whatever the engine's
    dtype."""

    in_names = ("in_proj",)
    out_name = "out_weight"

    def __init__(self, hidden_size: int, inner: int, state_size: int, dt_rank: int, conv_taps: int):
        self.hidden_size, self.inner, self.state_size = int(hidden_size), int(inner), int(state_size)
        self.dt_rank, self.conv_taps = int(dt_rank), int(conv_taps)
        self.ssm_floats = self.inner * self.state_size
        self.state_floats = self.ssm_floats + (self.conv_taps - 1) * self.inner

    def param_specs(self):
        I, N, R = self.inner, self.state_size, self.dt_rank
        return {"in_proj": ParamSpec((2 * I, self.hidden_size), "matrix"),
                "conv_weight": ParamSpec((I, self.conv_taps), "vector"), "conv_bias": ParamSpec((I,), "vector"),
                "x_proj": ParamSpec((R + 2 * N, I), "matrix"),
                "dt_weight": ParamSpec((I, R), "matrix"), "dt_bias": ParamSpec((I,), "vector"),
                "A_log": ParamSpec((I, N), "vector"), "D": ParamSpec((I,), "vector"),
                "out_weight": ParamSpec((self.hidden_size, I), "matrix")}

    def kernel_limits(self, dtype: str):
        from .. import ops
        out = []
        if not (1 <= self.state_size <= ops.SELECTIVE_MAX_STATE):
            out.append(f"mamba: a state of {self.state_size} entries per channel; the kernels take {ops.SELECTIVE_MAX_STATE}")
        if not (1 <= self.dt_rank <= ops.SELECTIVE_MAX_RANK):
            out.append(f"mamba: step sizes of rank {self.dt_rank}; the kernels take {ops.SELECTIVE_MAX_RANK}")
        if not (1 <= self.conv_taps <= ops.SSD_MAX_TAPS):
            out.append(f"mamba: a convolution of {self.conv_taps} taps; the kernel takes 1 to {ops.SSD_MAX_TAPS}")
        return out

    def cache_need(self):
        return StateNeed((self.state_floats,), "float32")

    def bind(self, params, rt) -> None:
        import torch
        super().bind(params, rt)
        if "A_log" in params:
            self.A = (-torch.exp(self.A_log.double())).float().contiguous()
            # rows of the step sizes' projection padded to 16-byte pieces; the padding is zero
            R8 = -(-self.dt_rank // 8) * 8
            padded = torch.zeros((self.inner, R8), dtype=self.dt_weight.dtype, device=self.dt_weight.device)
            padded[:, :self.dt_rank] = self.dt_weight
            self.dt_narrow = self.dt_weight         # as stored, for tables too narrow for the padded columns
            self.dt_weight = padded

    def core(self, proj, ctx, cache, out, out_scale: float = 1.0) -> None:
        import torch
        ops = self.rt.ops
        T, I, N, R = proj.shape[0], self.inner, self.state_size, self.dt_rank
        R8, wide = self.dt_weight.shape[1], R + 2 * N
        act = self.rt.act_dtype
        x = ctx.ws.buf("mamba_x", T, -(-I // 8) * 8, act)[:, :I]
        ops.ssd_conv(proj, 0, self.conv_weight, self.conv_bias, cache.state, self.ssm_floats, ctx, x, write_state=cache.write)
        low = ctx.ws.buf("mamba_low", T, max(R8, -(-wide // 8) * 8), act)     # rows stay 16-byte aligned
        ops.linear(x, self.x_proj, None, out=low[:, :wide])
        z = proj[:, I:2 * I]
        args = (z, self.A, self.D, self.dt_bias, cache.state, ctx, out)
        if getattr(ctx, "decode_only", False):
            ops.selective_step(x, low[:, :wide], R, R, R + N, self.dt_weight, *args, out_scale=out_scale, write_state=cache.write)
            return
        dt = ctx.ws.buf("mamba_dt", T, I, torch.float32)
        if R8 <= wide:          # the columns beyond the rank are B's: finite, and their weights are zero
            ops.linear(low[:, :R8], self.dt_weight, None, out=dt)
        else:
            ops.linear(low[:, :R], self.dt_narrow, None, out=dt)
        ops.selective_scan(x, dt, low, R, R + N, *args, out_scale=out_scale, write_state=cache.write)


register_part("mixer", "mamba", MambaMixer)

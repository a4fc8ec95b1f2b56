"""State-space duality (Mamba-2): a recurrent mixer whose decay is one number per head and token.

With H heads of ``vdim`` numbers, a state of N numbers per value column, G groups that share B and
C (head h uses group h // (H / G)), and the input projection's columns [z | x | B | C | dt]:

    x, B, C <- silu(conv(x), conv(B), conv(C))     causal, per channel, with a bias; the last tap
                                                   meets the current token
    dt_h    <- softplus(dt_h + dt_bias_h);   a_h = exp(-exp(A_log_h) dt_h)
    S_h     <- a_h S_h + dt_h B x_h^T ;   y_h = S_h^T C + D_h x_h
    out = W_o [ rms_parts(y * silu(z)) * norm ]    the gate before the norm, which is taken in
                                                   ``norm_groups`` equal parts of the row

Per request the cache keeps the float32 states [H, N, vdim] and behind them the convolutions'
newest inputs as a ring of ``taps`` rows (position p in row p % taps), so that a step of single
tokens can write the newest row while others still read the rows before it.  Decays, step sizes,
state, gate and norm are float32 in both precisions.  The state starts at zero (the runner clears
a slot when a request is opened) and is carried from step to step.
"""

from __future__ import annotations

import torch

from .base import Mixer, TensorRequest, register_mixer


class StateSpace(Mixer):
    writes_fresh = True

    def __init__(self, *, width: int, n_heads: int, vdim: int, state: int, groups: int, taps: int,
                 norm_groups: int, eps: float, prefix: str):
        if n_heads % groups:
            raise ValueError(f"n_heads {n_heads} is not a multiple of groups {groups}")
        if n_heads * vdim % norm_groups:
            raise ValueError(f"a row of {n_heads * vdim} numbers has no {norm_groups} equal parts")
        if taps < 1:
            raise ValueError("a short convolution has at least one tap")
        self.width, self.H, self.V, self.N, self.G = width, n_heads, vdim, state, groups
        self.taps, self.norm_groups = int(taps), int(norm_groups)
        self.eps, self.p = float(eps), prefix
        self.inner = self.H * self.V
        self.channels = self.inner + 2 * self.G * self.N              # x | B | C
        self.n_in = self.inner + self.channels + self.H               # z | x | B | C | dt
        self.sizes = dict(heads=self.H, groups=self.G, state_dim=self.N, vdim=self.V,
                          taps=self.taps)

    def tensor_requests(self):
        p, W, H, C = self.p, self.width, self.H, self.channels
        return {p + "in": TensorRequest((self.n_in, W), "matrix"),
                p + "conv": TensorRequest((C, self.taps), "float32"),
                p + "conv.b": TensorRequest((C,), "vector"),
                p + "dt_bias": TensorRequest((H,), "vector"),
                p + "A_log": TensorRequest((H,), "vector"), p + "D": TensorRequest((H,), "vector"),
                p + "norm": TensorRequest((self.inner,), "vector"),
                p + "o": TensorRequest((W, self.inner), "matrix")}

    def bind(self, tensors):
        p, t = self.p, tensors
        pad = -self.n_in % 8
        w = [t[p + "in"]] + ([t[p + "in"].new_zeros(pad, self.width)] if pad else [])
        self.w_in = torch.cat(w).contiguous()
        # tap by tap: neighbouring channels are neighbours
        self.conv_w, self.conv_b = t[p + "conv"].t().contiguous(), t[p + "conv.b"]
        self.dt_bias, self.a_log, self.skip = t[p + "dt_bias"], t[p + "A_log"], t[p + "D"]
        self.norm_w, self.w_out = t[p + "norm"], t[p + "o"]

    def state_shape(self):
        return (self.H * self.N * self.V + self.taps * self.channels,)

    def forward(self, ctx, h, x, cache, fresh=False):
        ops, T, C = ctx.ops, h.shape[0], self.channels
        proj = ctx.buffer("ssm_proj", (T, self.w_in.shape[0]), torch.float32)
        ops.linear(proj, h, self.w_in)
        y = ctx.buffer("ssm_y", (T, self.inner), torch.float32)
        state = ctx.state()
        conv = dict(conv_w=self.conv_w, conv_b=self.conv_b, dt_bias=self.dt_bias,
                    a_log=self.a_log, x_off=self.inner, **self.sizes)
        plan = getattr(ctx, "plan", None)
        if plan is not None and plan.single_new and plan.tile_cap == 0:
            # every request brings one token: convolutions, decay and state in one launch
            ops.ssm_step(y, state, proj, self.skip, ctx.tok_req, ctx.tok_pos, ctx.req_slot, **conv)
        else:
            wide = ops.ssm_rows_dtype(ctx.dtype, T, self.sizes)
            rows = ctx.buffer("ssm_rows", (T, C), wide)
            step = ctx.buffer("ssm_step", (T, 2 * self.H), torch.float32)
            ops.ssm_prepare(rows, step, proj, state, ctx.tok_req, ctx.tok_pos, ctx.req_start,
                            ctx.req_slot, **conv)
            ops.ssm_recurrence(y, state, rows, step, proj, self.skip, ctx.tok_pos, ctx.req_start,
                               ctx.req_len, ctx.req_slot, x_off=self.inner, **self.sizes)
        gated = ctx.buffer("ssm_gated", (T, self.inner), ctx.dtype)
        ops.head_norm_gate(gated, y, self.norm_w, proj, gate_offset=0, heads=self.norm_groups,
                           dim=self.inner // self.norm_groups, eps=self.eps, gate_act="silu",
                           gate_first=True)
        ops.linear(x, gated, self.w_out, None, residual=None if fresh else x)


register_mixer("state_space", StateSpace)

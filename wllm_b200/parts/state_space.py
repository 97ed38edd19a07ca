"""A state space with a scalar decay per head and token (Mamba-2).

'state_space': per head a state S [state_dim, value_dim] in 32-bit in the request's state slot (head h reads the B and C rows of group
h // (num_heads / groups)):

    S_t = exp(-exp(decay_log_h) dt_t) S_(t-1) + dt_t B_t x_t^T,    y_t = S_t^T C_t + skip_h x_t

in_proj x is z | x | B | C | dt (inner = num_heads * value_dim, inner, groups * state_dim twice, num_heads columns).  x, B and C pass a
causal convolution along the sequence, channel by channel (conv [channels, conv_taps], the last tap weighs the token itself, inputs in front
of the sequence count as zero; conv_bias; the newest conv_taps - 1 inputs are kept as state), and SiLU; dt = softplus(dt + step_bias).  y times
silu(z) is divided by its root mean square in norm_groups equal parts of the row, each by its own (eps), times the gain norm_weight [inner];
then o_proj.
spec options: num_heads, groups, state_dim, value_dim, conv_taps, norm_groups, eps, in_proj, conv, conv_bias (None: no bias), decay_log,
step_bias, skip, norm_weight, o_proj (checkpoint names).

Steps, decays and state are 32-bit (csrc/state_space.cu).  The recurrence is the decayed-state scan of csrc/linear_attention.cu with q = C,
k = B, v = x, whose long portions run in segments side by side, and, under bfloat16 in steps with portions of `SSD_CHUNKS_FROM` tokens and
more, a form in chunks on the tensor cores, which takes x, B and C in bfloat16.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import MIXERS, CacheRef, ParamSpec, StateNeed, as_branch


@MIXERS.register("state_space")
class StateSpace:
    graph_safe = True

    def __init__(self, spec, hidden_size: int, model_dtype: torch.dtype):
        self.heads, self.groups = int(spec.num_heads), int(spec.options.get("groups") or 1)
        self.state_dim, self.vdim, self.taps = int(spec.state_dim), int(spec.value_dim), int(spec.conv_taps)
        self.norm_groups, self.eps = int(spec.options.get("norm_groups") or 1), float(spec.eps)
        self.inner = self.heads * self.vdim
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError(f"{self.heads} heads in {self.groups} groups, rows of {self.inner} in {self.norm_groups} parts: no such cut")
        if self.state_dim > 256 or not 1 <= self.taps <= 16:
            raise ValueError(f"state_dim {self.state_dim}, conv_taps {self.taps}: the kernels hold states of up to 256 rows and convolutions of "
                             f"up to 16 taps")
        self.channels = self.inner + 2 * self.groups * self.state_dim
        self.width = self.inner + self.channels + self.heads
        self.hidden_size, self.model_dtype = hidden_size, model_dtype
        self.chunks = model_dtype == torch.bfloat16 and ops.ssd_chunks_ok(self.heads, self.state_dim, self.vdim)
        self.names = {k: spec.options[k] for k in ("in_proj", "conv", "decay_log", "step_bias", "skip", "norm_weight", "o_proj")}
        self.bias_name = spec.options.get("conv_bias")
        self.tag = ""
        self.w_in = self.wo = self.conv = self.conv_bias = self.a_log = self.dt_bias = self.skip = self.gain = None

    def cache_need(self):
        need = [("state", (self.heads, self.state_dim, self.vdim), torch.float32)]
        if self.taps > 1:
            need.append(("conv", (self.taps - 1, self.channels), torch.float32))
        return StateNeed(tuple(need))

    def param_specs(self):
        H, n = self.hidden_size, self.names
        out = [ParamSpec(n["in_proj"], (self.width, H)), ParamSpec(n["conv"], (self.channels, self.taps))]
        if self.bias_name is not None:
            out.append(ParamSpec(self.bias_name, (self.channels,), "vector"))
        return out + [ParamSpec(n[k], (self.heads,), "vector") for k in ("step_bias", "decay_log", "skip")] + \
            [ParamSpec(n["norm_weight"], (self.inner,), "vector"), ParamSpec(n["o_proj"], (H, self.inner))]

    def load(self, fetch):
        n = self.names
        def wide(name):
            return fetch(name).to(torch.float32).contiguous()
        w = fetch(n["in_proj"])
        pad = -self.width % 8             # the product's rows in steps of 8 columns (16 bytes of the matrix type)
        self.w_in = (torch.cat([w, w.new_zeros((pad, self.hidden_size))], dim=0) if pad else w).contiguous()
        self.conv, self.a_log, self.dt_bias = wide(n["conv"]), wide(n["decay_log"]), wide(n["step_bias"])
        self.conv_bias = wide(self.bias_name) if self.bias_name is not None else None
        self.gain = fetch(n["norm_weight"]).contiguous()
        self.skip = fetch(n["skip"]).to(self.gain.dtype).contiguous()
        self.wo = fetch(n["o_proj"]).contiguous()

    def input_weights(self) -> list:
        return [self.w_in]

    def __call__(self, x: torch.Tensor, ctx, cache: CacheRef):
        fused, parts = ops.project(x, self.w_in, lambda name, shape, dt: ctx.buffer(self.tag + "ssd_in_" + name, shape, dt))
        return self.mix(fused, parts, 0, ctx, cache)

    def mix(self, fused: torch.Tensor, parts: int, col0: int, ctx, cache: CacheRef):
        """The mixer on the columns from col0 of a fused product [n, W] (or partial sums [parts, n, W])."""
        n, H, N, V, f32 = fused.shape[-2], self.heads, self.state_dim, self.vdim, torch.float32
        inner, rows = self.inner, self.groups * self.state_dim
        chunked = self.chunks and ctx.max_q_len >= ops.SSD_CHUNKS_FROM
        xbc = ctx.buffer(self.tag + "ssd_xbc", (n, self.channels), self.model_dtype if chunked else f32)
        pairs = ctx.buffer(self.tag + "ssd_pairs", (n, H, 2), f32)
        conv_state = ctx.state(cache.state_names["conv"]) if self.taps > 1 else None
        single = ctx.num_multi == 0              # no request brings more than one token
        ops.ssd_prepare(fused, parts, col0 + inner, col0 + inner + self.channels, self.taps, self.conv, self.conv_bias, self.a_log,
                        self.dt_bias, ctx, conv_state, xbc, pairs, shift=single)
        if self.taps > 1 and not single:
            ops.ssd_conv_update(fused, parts, col0 + inner, self.taps, ctx, conv_state)
        x, b, c = xbc[:, :inner], xbc[:, inner:inner + rows], xbc[:, inner + rows:]
        o = ctx.buffer(self.tag + "ssd_o", (n, inner), f32)
        state, share = ctx.state(cache.state_names["state"]), H // self.groups
        if chunked:
            ops.ssd_chunks(xbc, pairs, state, o, ctx.req_q_start, ctx.req_q_len, ctx.req_slot, H, share, N, V)
        else:
            seg_len, max_seg = ops.linattn_segment_plan(ctx.max_q_len, ctx.num_multi, H, V)
            seg_state = seg_decay = None
            if max_seg > 1:
                R = ctx.n_requests
                seg_state = ctx.buffer(self.tag + "ssd_seg_state", (R * max_seg * H * N * V,), f32)
                seg_decay = ctx.buffer(self.tag + "ssd_seg_decay", (R * max_seg * H * N,), f32)
            ops.linattn_scan(c, b, x, None, None, state, o, ctx.req_q_start, ctx.req_q_len, ctx.req_slot, H, N, V, seg_len, max_seg, seg_state,
                             seg_decay, pairs=pairs, share=share)
        gated = ctx.buffer(self.tag + "ssd_gated", (n, inner), self.model_dtype)
        ops.ssd_gate_norm(o, x, self.skip, fused, parts, col0, self.gain, self.eps, gated, self.norm_groups)
        return as_branch(ops.project(gated, self.wo, lambda name, shape, dt: ctx.buffer(self.tag + "ssd_out_" + name, shape, dt)))

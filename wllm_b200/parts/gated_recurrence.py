"""A gated linear recurrent unit behind a short convolution.

'rg_lru': two branches of `width` channels, y = gelu_tanh(y_proj x + y_bias) and u = conv(x_proj x + x_bias), a causal convolution per
channel with `conv_taps` taps that look back only (the last tap weighs the token itself; inputs in front of the sequence are zero)
and a bias; u in `blocks` equal parts, each with two square maps,

    r = sigmoid(r_gate u + r_bias),  i = sigmoid(i_gate u + i_bias),  log a = -c r softplus(decay),  a = exp(log a)
    S_t = a S_(t-1) + sqrt(1 - a^2) i u,    output = o_proj(S * y)

S starts at zero and lives, per channel, in 32-bit in the request's state slot, beside the convolution's last inputs (a ring of
conv_taps rows, the input of position p in row p mod conv_taps).  Convolution, gates and recurrence are 32-bit (csrc/rg_lru.cu).

spec options: width, blocks, conv_taps, gate_factor (c), y_proj / x_proj [width, hidden], y_bias, x_bias [width], conv [width,
conv_taps], conv_bias [width], r_gate / i_gate [blocks, width / blocks, width / blocks] (out, in), r_bias / i_bias [blocks, width /
blocks], decay [width], o_proj [hidden, width] (checkpoint names).  One product makes y | x.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import MIXERS, CacheRef, ParamSpec, StateNeed, as_branch

_NAMES = ("y_proj", "x_proj", "y_bias", "x_bias", "conv", "conv_bias", "r_gate", "i_gate", "r_bias", "i_bias", "decay", "o_proj")


@MIXERS.register("rg_lru")
class GatedRecurrence:
    graph_safe = True

    def __init__(self, spec, hidden_size: int, model_dtype: torch.dtype):
        self.width, self.blocks, self.taps = int(spec.width), int(spec.blocks), int(spec.conv_taps)
        if self.width % self.blocks:
            raise ValueError(f"{self.width} channels in {self.blocks} equal blocks: no such cut")
        self.c = float(spec.gate_factor)
        self.hidden_size, self.model_dtype = hidden_size, model_dtype
        self.names = {k: spec.options[k] for k in _NAMES}
        self.w_in = self.wo = self.conv = self.conv_bias = self.x_bias = self.y_bias = None
        self.maps = self.ra_bias = self.ri_bias = self.rate = None
        self.x_off = 0
        self.tag = ""

    def cache_need(self):
        return StateNeed((("state", (self.width,), torch.float32), ("conv", (self.taps, self.width), torch.float32)))

    def param_specs(self):
        H, W, B, n = self.hidden_size, self.width, self.blocks, self.names
        s = W // B
        return [ParamSpec(n["y_proj"], (W, H)), ParamSpec(n["y_bias"], (W,), "vector"), ParamSpec(n["x_proj"], (W, H)),
                ParamSpec(n["x_bias"], (W,), "vector"), ParamSpec(n["conv"], (W, self.taps)), ParamSpec(n["conv_bias"], (W,), "vector"),
                ParamSpec(n["r_gate"], (B, s, s)), ParamSpec(n["r_bias"], (B, s), "vector"), ParamSpec(n["i_gate"], (B, s, s)),
                ParamSpec(n["i_bias"], (B, s), "vector"), ParamSpec(n["decay"], (W,), "vector"), ParamSpec(n["o_proj"], (H, W))]

    def load(self, fetch):
        n = self.names
        def vector(name):
            return fetch(n[name]).to(torch.float32).reshape(-1).contiguous()
        y = fetch(n["y_proj"])
        pad = -self.width % 8                 # x's columns begin on a multiple of 8 (16 bytes of the matrix type), and so do the rows
        gap = [y.new_zeros((pad, self.hidden_size))] if pad else []
        self.x_off = self.width + pad
        self.w_in = torch.cat([y] + gap + [fetch(n["x_proj"])] + gap, dim=0).contiguous()
        self.wo = fetch(n["o_proj"]).contiguous()
        self.conv = fetch(n["conv"]).to(torch.float32).t().contiguous()
        self.x_bias, self.y_bias, self.conv_bias = vector("x_bias"), vector("y_bias"), vector("conv_bias")
        # log a = -rate r: what the gate does not touch is worked out once (in 64-bit, rounded once)
        self.rate = (self.c * torch.nn.functional.softplus(fetch(n["decay"]).to(torch.float64))).to(torch.float32).contiguous()
        # both gates' rows of a block one below the other; in bfloat16 each row twice side by side, for the two pieces of u
        maps = torch.cat([fetch(n["r_gate"]), fetch(n["i_gate"])], dim=1)
        self.maps = (torch.cat([maps, maps], dim=2) if self.model_dtype == torch.bfloat16 else maps).contiguous()
        self.ra_bias, self.ri_bias = vector("r_bias"), vector("i_bias")

    def __call__(self, x: torch.Tensor, ctx, cache: CacheRef):
        n, W = x.shape[0], self.width
        fused, parts = ops.project(x, self.w_in, lambda name, shape, dt: ctx.buffer(self.tag + "lru_in_" + name, shape, dt))
        unit = dict(y_off=0, x_off=self.x_off, x_bias=self.x_bias, y_bias=self.y_bias, taps=self.conv, conv_bias=self.conv_bias)
        gates = dict(maps=self.maps, ra_bias=self.ra_bias, ri_bias=self.ri_bias, rate=self.rate)
        state, ring = ctx.state(cache.state_names["state"]), ctx.state(cache.state_names["conv"])
        out = ctx.buffer(self.tag + "lru_out", (n, W), self.model_dtype)
        if ctx.num_multi == 0 and self.model_dtype == torch.bfloat16 and ops.rglru_step_ok(gates, fused, self.x_off):
            ops.rglru_step(fused, parts, unit, gates, ctx, ring, state, out)
        else:
            if n >= ops.RGLRU_GROUPED_FROM and ops.rglru_grouped_ok(gates, fused, self.x_off):
                B, rows = self.blocks, self.maps.shape[1]
                uv = ctx.buffer(self.tag + "lru_pieces", (B * n, rows), torch.bfloat16)
                z = ctx.buffer(self.tag + "lru_gate_sums", (B * n, rows), torch.float32)
                tiles = ctx.buffer(self.tag + "lru_tiles", (1 + 3 * ops.moe_row_tiles(B * n, B),), torch.int32)
                ops.rglru_gate_sums(fused, parts, unit, gates, ctx, ring, uv, tiles, z)
                pairs = (z, uv)
            else:
                pairs = ctx.buffer(self.tag + "lru_pairs", (n, W, 2), torch.float32)
                ops.rglru_gates(fused, parts, unit, gates, ctx, ring, pairs)
            ops.rglru_scan(fused, parts, unit, gates, ctx, ring, pairs, state, out, ctx.max_q_len >= ops.RGLRU_RUNS_FROM)
        return as_branch(ops.project(out, self.wo, lambda name, shape, dt: ctx.buffer(self.tag + "lru_branch_" + name, shape, dt)))

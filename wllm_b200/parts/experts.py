"""Routed experts: a feed-forward in which every token runs a few of many small gated units.

spec options: num_experts, top, groups, groups_kept (the experts form `groups` equal groups of neighbours; a group's score
is its best expert's and only experts of the `groups_kept` best groups can be chosen; 1 and 1: no such limit), router
(checkpoint name of the router matrix [experts, hidden]), expert_prefix (expert j's tensors are <prefix><j>.gate / .up /
.down), intermediate_size, activation, limit, slope (the experts' gated unit, as 'gated_dense' takes them), scores ('softmax',
the default, over all experts; 'sigmoid': expert by expert, not normalised), gated (default True; False: an expert is
down(act(up x)) with tensors <prefix><j>.up / .down and activation 'relu_squared'), weight_on ('output', the default: the
chosen experts' outputs are multiplied by their scores; 'input': their inputs are, the output is the sum of expert(s x)), shared (None, or
the options of a 'gated_dense' unit that every token runs, plus gate_weight: the checkpoint name of one row [1, hidden], the
unit's output is multiplied by sigmoid(row . x); without gate_weight it is added as it is), identity (so many further experts behind the
num_experts, without tensors, whose output is the token's row itself; the router has a row for each), correction (checkpoint
name of a vector [num_experts + identity] that joins the scores for the choice alone), renorm_eps (the weights are the chosen
scores over their sum + renorm_eps; absent: the scores as they are), router_bias (checkpoint name of a vector [num_experts + identity]
added to the router's logits).  scores may also be 'softmax_chosen': the `top` largest logits are chosen and weighted by the softmax
over the chosen logits alone (no groups, correction or renorm_eps).  A gated expert's activation is 'capped_swish' (limit, slope) or
'silu' (down(silu(gate x) * up x), no limit or slope).

Router logits, the softmax over all experts, the choice and the weights (the chosen experts' scores as they are) are
32-bit, against a 32-bit copy of the router matrix.  The tokens' (token, rank) pairs are sorted by expert on the device
and the experts run as two grouped products over the sorted rows (csrc/moe.cu; from `TC_FROM_PAIRS` pairs on, under
bfloat16, on the grouped form of the tensor-memory product, csrc/gemm_bf16_tc.cu); a token's output is the sum over its
ranks in rank order, so it does not depend on the batch beyond the rounding of the products.  Nothing comes back to the host, and every launch is sized
from the number of tokens and experts alone.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import FEED_FORWARDS, ParamSpec, branch_pair, spec as make_spec


@FEED_FORWARDS.register("routed_experts")
class RoutedExperts:
    graph_safe = True
    TC_FROM_PAIRS = 1024       # (token, expert) pairs from which the experts' products run on the tensor-memory kernel

    def __init__(self, spec, hidden_size: int, model_dtype: torch.dtype):
        self.E, self.top = int(spec.num_experts), int(spec.top)
        self.identity = int(spec.options.get("identity") or 0)
        self.slots = self.E + self.identity                       # what the router chooses from
        self.correction_name, self.renorm_eps = spec.options.get("correction"), spec.options.get("renorm_eps")
        self.groups, self.groups_kept = int(spec.options.get("groups") or 1), int(spec.options.get("groups_kept") or 1)
        if self.slots % self.groups or not 1 <= self.groups_kept <= self.groups or not 1 <= self.top <= self.groups_kept * (self.slots // self.groups):
            raise ValueError(f"{self.slots} experts in {self.groups} groups, {self.groups_kept} kept, top {self.top}: no such choice")
        self.inter, self.activation = int(spec.intermediate_size), spec.activation
        self.gated = bool(spec.options.get("gated", True))
        self.scores, self.weight_on = spec.options.get("scores") or "softmax", spec.options.get("weight_on") or "output"
        if self.scores not in ops.ROUTER_SCORES or self.weight_on not in ("output", "input"):
            raise ValueError(f"scores {self.scores!r} ({', '.join(ops.ROUTER_SCORES)}), weight_on {self.weight_on!r} ('output', 'input')")
        if self.scores == "softmax_chosen" and (self.groups > 1 or self.correction_name is not None or self.renorm_eps is not None):
            raise ValueError("a softmax over the chosen logits knows no groups, no correction and no division by the scores' sum")
        if self.activation not in (ops.EXPERT_GATED_UNITS if self.gated else ("relu_squared",)):
            raise ValueError(f"the grouped expert products are built for gated experts with the activation {' or '.join(ops.EXPERT_GATED_UNITS)} "
                             "and for experts without a gate with relu_squared")
        if self.weight_on == "input" and self.identity:
            raise ValueError("scores on the experts' inputs are built without identity experts")
        if self.weight_on == "input" and self.gated:
            raise ValueError("scores on the experts' inputs are built for experts without a gate")
        self.limit, self.slope = float(spec.options.get("limit") or 0.0), float(spec.options.get("slope") or 0.0)
        self.router_name, self.prefix, self.bias_name = spec.router, spec.expert_prefix, spec.options.get("router_bias")
        self.hidden_size, self.model_dtype = hidden_size, model_dtype
        self.shared = self.gate_name = None
        shared = spec.options.get("shared")
        if shared is not None:
            shared = dict(shared)
            self.gate_name = shared.pop("gate_weight", None)
            self.shared = FEED_FORWARDS.build(make_spec("gated_dense", **shared), hidden_size=hidden_size, model_dtype=model_dtype)
        self.w_router = self.w_gate = self.w_gu = self.w_down = self.correction = self.router_bias = None

    def parts(self):
        return [] if self.shared is None else [self.shared]

    def param_specs(self):
        H, I = self.hidden_size, self.inter
        out = [ParamSpec(self.router_name, (self.slots, H))]
        if self.correction_name is not None:
            out.append(ParamSpec(self.correction_name, (self.slots,), "vector"))
        if self.bias_name is not None:
            out.append(ParamSpec(self.bias_name, (self.slots,), "vector"))
        for j in range(self.E):
            p = f"{self.prefix}{j}."
            out += ([ParamSpec(p + "gate", (I, H))] if self.gated else []) + [ParamSpec(p + "up", (I, H)), ParamSpec(p + "down", (H, I))]
        if self.shared is not None:
            out += self.shared.param_specs() + ([ParamSpec(self.gate_name, (1, H))] if self.gate_name is not None else [])
        return out

    def load(self, fetch):
        self.w_router = fetch(self.router_name).to(torch.float32).contiguous()
        if self.correction_name is not None:
            self.correction = fetch(self.correction_name).to(torch.float32).contiguous()
        if self.bias_name is not None:
            self.router_bias = fetch(self.bias_name).to(torch.float32).contiguous()
        names = [f"{self.prefix}{j}." for j in range(self.E)]
        if self.gated:
            self.w_gu = torch.stack([torch.cat([fetch(p + "gate"), fetch(p + "up")], dim=0) for p in names]).contiguous()
        else:
            self.w_gu = torch.stack([fetch(p + "up") for p in names]).contiguous()
        self.w_down = torch.stack([fetch(p + "down") for p in names]).contiguous()
        if self.shared is not None:
            self.shared.load(fetch)
        if self.gate_name is not None:
            self.w_gate = fetch(self.gate_name).to(torch.float32).reshape(-1).contiguous()

    def __call__(self, x: torch.Tensor, ctx):
        n, top, H = x.shape[0], self.top, self.hidden_size
        pairs = n * top
        chosen = ctx.buffer("moe_chosen", (n, top), torch.int32)
        weights = ctx.buffer("moe_weights", (n, top), torch.float32)
        gate = ctx.buffer("moe_gate", (n,), torch.float32) if self.gate_name is not None else None
        ops.moe_route(x, self.w_router, self.w_gate, chosen, weights, gate, self.groups, self.groups_kept, scores=self.scores,
                      correction=self.correction, renorm_eps=self.renorm_eps, bias=self.router_bias)
        unit = None if self.activation == "capped_swish" else self.activation
        on_input = weights.view(-1) if self.weight_on == "input" else None
        slots = self.slots
        index = ctx.buffer("moe_index", (2 * slots + 1 + 2 * pairs,), torch.int32)
        count, offset = index[:slots], index[slots:2 * slots + 1]
        order, place = index[2 * slots + 1:2 * slots + 1 + pairs], index[2 * slots + 1 + pairs:]
        real = offset[:self.E + 1]          # identity experts' pairs lie behind all others: the products see the first E experts
        act = ctx.buffer("moe_act", (pairs, self.inter), self.model_dtype)
        y = ctx.buffer("moe_y", (pairs, H), torch.float32)
        # Many rows (portions of prompts): the products run on the tensor-memory kernel over row tiles of one expert each, on
        # the tokens' rows copied into sorted order.  Few rows (decoding) are bound by streaming the experts' weights, which
        # the kernel on mma.sync does from rows gathered on the fly.
        if pairs >= self.TC_FROM_PAIRS and x.dtype == torch.bfloat16 and ops.tc_grouped_ok(x, self.w_gu) and self.inter % 8 == 0:
            tiles = ctx.buffer("moe_tiles", (1 + 3 * ops.moe_row_tiles(pairs, self.E),), torch.int32)
            ops.moe_plan(chosen, count, offset, order, place, tiles, ctx.buffer("moe_plan", (ops.MOE_PLAN_SEGMENTS * slots,), torch.int32),
                         real_experts=self.E)
            # (scores on the inputs: the rows are multiplied while they are copied, rounded once)
            rows = ops.moe_gather(x, order, top, ctx.buffer("moe_rows", (pairs, H), self.model_dtype), row_weights=on_input)
            ops.gemm_bf16_tc_grouped(rows, self.w_gu, act, tiles, self.gated, self.limit, self.slope, unit=unit)
            ops.gemm_bf16_tc_grouped(act, self.w_down, y, tiles, False)
        else:
            ops.moe_plan(chosen, count, offset, order, place)
            # (scores on the inputs: the up product is linear, so the score multiplies its 32-bit sums in front of the activation)
            ops.moe_grouped(x, self.w_gu, act, real, order, top, self.gated, self.limit, self.slope, unit=unit, row_weights=on_input)
            ops.moe_grouped(act, self.w_down, y, real, order, top, False)
        shared = branch_pair(self.shared(x, ctx)) if self.shared is not None else None
        out = ctx.buffer("moe_out", (n, H), torch.float32)
        own = dict(chosen=chosen, real_experts=self.E, x=x) if self.identity else {}
        return ops.moe_combine(y, place, None if self.weight_on == "input" else weights, shared, gate, out, **own)

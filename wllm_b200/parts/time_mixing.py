"""Time mixing over blends of neighbouring tokens, and two mixers side by side whose outputs are added with factors.

'time_mixing': with h' the row of the token before (zeros in front of the sequence), every stream s of r, k, v, g, w reads its own
blend h + (h' - h) * mu_s.  r, k, v are projections of theirs (num_heads heads of key_dim); the decay of every head and key channel is
exp(-exp(decay_up tanh(decay_down blend_w) + decay_bias)); per head a state S [key_dim, key_dim] in 32-bit in the request's state slot,

    o_t = (S_(t-1) + diag(bonus) k_t v_t^T)^T r_t,    S_t = diag(decay_t) S_(t-1) + k_t v_t^T

Each head's o is divided by its root mean square (eps); the row of all heads is multiplied by the gain `norm_weight`
[num_heads * key_dim] and by silu(g_proj blend_g), and projected.  The last row of every portion is kept as state (two rows, the row of
position p in row p mod 2).
spec options: num_heads, key_dim, eps, mu_r / mu_k / mu_v / mu_g / mu_w, r_proj / k_proj / v_proj / g_proj [heads * key_dim, hidden],
decay_down [rank, hidden], decay_up [heads * key_dim, rank], decay_bias, bonus [heads, key_dim], norm_weight, o_proj (checkpoint names),
rank (absent: the checkpoint's).

'parallel_sum': left_factor * left(x) + right_factor * right(x).  The left mixer is an 'attention', the right one a 'time_mixing'; their
heads lie side by side in one row (the right one's already times right_factor / left_factor, in 32-bit) and one output product takes
both; left_factor is left to whoever folds the branch into the residual.  Steps of single tokens under bfloat16 make all
products that read x, or a blend of it, in one kernel (csrc/token_blend.cu).  Portions blend first; r, k, v and g are then one
grouped product on the tensor cores.
spec options: left, right (mixer specs), left_factor, right_factor.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import MIXERS, BranchSum, CacheRef, KVNeed, ParamSpec, StateNeed, as_branch
from .linear_attention import ParallelMean

STREAMS = "rkvgw"


@MIXERS.register("time_mixing")
class TimeMixing:
    graph_safe = True

    def __init__(self, spec, hidden_size: int, model_dtype: torch.dtype):
        self.heads, self.dim = int(spec.num_heads), int(spec.key_dim)
        if self.dim > 256:
            raise ValueError(f"key_dim {self.dim}: the recurrence kernel holds up to 256 key channels a head")
        self.eps = float(spec.eps)
        self.rank = spec.options.get("rank")
        self.hidden_size, self.model_dtype = hidden_size, model_dtype
        self.names = {k: spec.options[k] for k in [f"mu_{s}" for s in STREAMS] + ["r_proj", "k_proj", "v_proj", "g_proj", "decay_down",
                                                                                  "decay_up", "decay_bias", "bonus", "norm_weight", "o_proj"]}
        self.mu = self.w_rkvg = self.w_down = self.w_up = self.b_up = self.bonus = self.gain = self.wo = None
        self.tag = ""

    @property
    def out_width(self) -> int:
        return self.heads * self.dim

    def cache_need(self):
        return StateNeed((("state", (self.heads, self.dim, self.dim), torch.float32), ("row", (2, self.hidden_size), self.model_dtype)))

    def param_specs(self):
        H, HD, n = self.hidden_size, self.out_width, self.names
        return [ParamSpec(n[f"mu_{s}"], (H,), "vector") for s in STREAMS] + [ParamSpec(n[k], (HD, H)) for k in ("r_proj", "k_proj", "v_proj", "g_proj")] + \
            [ParamSpec(n["decay_down"], (self.rank, H)), ParamSpec(n["decay_up"], (HD, self.rank)), ParamSpec(n["decay_bias"], (HD,), "vector"),
             ParamSpec(n["bonus"], (self.heads, self.dim), "vector"), ParamSpec(n["norm_weight"], (HD,), "vector"), ParamSpec(n["o_proj"], (H, HD))]

    def load(self, fetch):
        n = self.names
        self.mu = torch.stack([fetch(n[f"mu_{s}"]).to(torch.float32) for s in STREAMS]).contiguous()
        self.w_rkvg = torch.stack([fetch(n[k]) for k in ("r_proj", "k_proj", "v_proj", "g_proj")]).contiguous()
        self.w_down, self.w_up = fetch(n["decay_down"]).contiguous(), fetch(n["decay_up"]).contiguous()
        self.rank = int(self.w_down.shape[0])
        if self.w_up.shape[1] != self.rank:
            raise ValueError(f"{n['decay_down']} has {self.rank} rows, {n['decay_up']} reads {self.w_up.shape[1]}")
        self.b_up = fetch(n["decay_bias"]).to(self.w_up.dtype).contiguous()
        self.bonus = fetch(n["bonus"]).to(torch.float32).reshape(-1).contiguous()
        self.gain = fetch(n["norm_weight"]).contiguous()
        self.wo = fetch(n["o_proj"]).contiguous()

    def projections(self, x: torch.Tensor, ctx, cache: CacheRef) -> tuple:
        """(r, k, v, g [n, heads * key_dim], low, parts of low): the blends of a step's rows and their products."""
        n, H, HD, tag = x.shape[0], self.hidden_size, self.out_width, self.tag
        blends = ctx.buffer(tag + "tm_blends", (len(STREAMS), n, H), self.model_dtype)
        kept = ctx.state(cache.state_names["row"])
        flat = blends[:4].view(4 * n, H)
        if ops.tc_grouped_ok(flat, self.w_rkvg):
            tiles = ctx.buffer(tag + "tm_tiles", (1 + 3 * ops.moe_row_tiles(4 * n, 4),), torch.int32)
            ops.token_blend(x, self.mu, ctx, kept, blends, tiles, 4)
            rkvg = ctx.buffer(tag + "tm_rkvg", (4 * n, HD), torch.float32)
            ops.gemm_bf16_tc_grouped(flat, self.w_rkvg, rkvg, tiles, False)
            r, k, v, g = (rkvg[i * n:(i + 1) * n] for i in range(4))
        else:
            ops.token_blend(x, self.mu, ctx, kept, blends)
            r, k, v, g = (ops.linear(blends[i], self.w_rkvg[i], ctx.buffer(tag + f"tm_{STREAMS[i]}", (n, HD), torch.float32), f32_out=True)
                          for i in range(4))
        low, parts = ops.project(blends[4], self.w_down, lambda name, shape, dt: ctx.buffer(tag + "tm_low_" + name, shape, dt))
        return r, k, v, g, low, parts

    def recur(self, r, k, v, g, low, low_parts: int, low_off: int, ctx, cache: CacheRef, out: torch.Tensor, factor: float = 1.0) -> None:
        """Decay, recurrence, head norm, gain and gate: what the output projection reads, times `factor`, into `out` [n, heads * key_dim]."""
        n, H, D, f32 = r.shape[0], self.heads, self.dim, torch.float32
        decay = ops.linattn_decay(low, low_parts, low_off, self.w_up, self.b_up, H, D, ctx.buffer(self.tag + "tm_decay", (n, H * D), f32))
        o = ctx.buffer(self.tag + "tm_o", (n, H * D), f32)
        seg_len, max_seg = ops.linattn_segment_plan(ctx.max_q_len, ctx.num_multi, H, D)
        seg_state = seg_decay = None
        if max_seg > 1:
            R = ctx.n_requests
            seg_state = ctx.buffer(self.tag + "tm_seg_state", (R * max_seg * H * D * D,), f32)
            seg_decay = ctx.buffer(self.tag + "tm_seg_decay", (R * max_seg * H * D,), f32)
        ops.linattn_scan(r, k, v, decay, None, ctx.state(cache.state_names["state"]), o, ctx.req_q_start, ctx.req_q_len, ctx.req_slot,
                         H, D, D, seg_len, max_seg, seg_state, seg_decay, bonus=self.bonus)
        ops.head_gate_norm(o, g, 0, 0, self.gain, self.eps, out, H, D, factor)

    def __call__(self, x: torch.Tensor, ctx, cache: CacheRef):
        out = ctx.buffer(self.tag + "tm_gated", (x.shape[0], self.out_width), self.model_dtype)
        r, k, v, g, low, parts = self.projections(x, ctx, cache)
        self.recur(r, k, v, g, low, parts, 0, ctx, cache, out)
        return as_branch(ops.project(out, self.wo, lambda name, shape, dt: ctx.buffer(self.tag + "tm_branch_" + name, shape, dt)))


@MIXERS.register("parallel_sum")
class ParallelSum:
    graph_safe = True

    def __init__(self, spec, hidden_size: int, model_dtype: torch.dtype):
        kw = dict(hidden_size=hidden_size, model_dtype=model_dtype)
        self.left, self.right = MIXERS.build(spec.left, **kw), MIXERS.build(spec.right, **kw)
        if not hasattr(self.left, "heads") or not hasattr(self.right, "recur"):
            raise TypeError(f"mixers added with factors: an attention mixer and a time mixing, not {type(self.left).__name__} and {type(self.right).__name__}")
        for side, m in (("left", self.left), ("right", self.right)):
            m.tag = side + "_"
        if "o" in (getattr(self.left, "bias_names", None) or {}):
            raise ValueError("mixers that share an output product have no bias on it")
        self.left_factor, self.right_factor = float(spec.left_factor), float(spec.right_factor)
        self.hidden_size, self.model_dtype = hidden_size, model_dtype
        self.w_in = self.w_left = self.w_out = self.mu = None

    def parts(self):
        return [self.left, self.right]

    def cache_need(self):
        out = []
        for side, m in (("left", self.left), ("right", self.right)):
            need = m.cache_need()
            for one in need if isinstance(need, (tuple, list)) else (need,):
                if isinstance(one, StateNeed):
                    one = StateNeed(tuple((f"{side}.{name}", shape, dt) for name, shape, dt in one.tensors))
                out.append(one)
        if sum(isinstance(one, KVNeed) for one in out) > 1:
            raise ValueError("two mixers side by side that both read pages are not supported")
        return tuple(out)

    def param_specs(self):
        return self.left.param_specs() + self.right.param_specs()

    def load(self, fetch):
        self.left.load(fetch)
        self.right.load(fetch)
        r = self.right
        self.left_width, self.left_out = self.left.wqkv.shape[0], self.left.wo.shape[1]
        # every matrix that reads x or a blend of it, one below the other: the sides' own are views of it
        self.w_in = torch.cat([self.left.wqkv, r.w_rkvg.view(-1, self.hidden_size), r.w_down], dim=0).contiguous()
        HD = r.out_width
        self.segments = [(self.left_width, -1)] + [(HD, s) for s in range(4)] + [(r.rank, 4)]
        self.left.wqkv = None
        self.w_left = self.w_in[:self.left_width]
        r.w_rkvg = self.w_in[self.left_width:self.left_width + 4 * HD].view(4, HD, self.hidden_size)
        r.w_down = self.w_in[self.left_width + 4 * HD:]
        # one output product for both sides' heads.  left_factor is applied behind it; the right side's heads carry the ratio
        w_left = self.left.wo
        self.factor, self.ratio = self.left_factor, 0.0
        if self.left_factor == 0.0:
            w_left, self.factor, self.ratio = torch.zeros_like(w_left), self.right_factor, 1.0
        else:
            self.ratio = self.right_factor / self.left_factor
        pad = -(self.left_out + HD) % 8          # rows in steps of 8 elements; the columns behind the heads hold zeros
        self.both_width = self.left_out + HD + pad
        cols = [w_left, r.wo] + ([w_left.new_zeros((self.hidden_size, pad))] if pad else [])
        self.w_out = torch.cat(cols, dim=1).contiguous()
        self.left.wo = r.wo = None

    def __call__(self, x: torch.Tensor, ctx, cache: CacheRef):
        n, r = x.shape[0], self.right
        left_cache, right_cache = ParallelMean._side(cache, "left"), ParallelMean._side(cache, "right")
        both = ctx.buffer("parallel_heads", (n, self.both_width), self.model_dtype)
        lo, HD = self.left_out, r.out_width
        heads_left, heads_right = both[:, :lo], both[:, lo:lo + HD]
        if self.both_width > lo + HD:
            both[:, lo + HD:].zero_()
        if ctx.num_multi == 0 and ops.blended_product_ok(x, self.w_in):
            fused = ctx.buffer("parallel_in", (n, self.w_in.shape[0]), torch.float32)
            ops.blended_product(x, r.mu, self.w_in, self.segments, ctx, ctx.state(right_cache.state_names["row"]), fused)
            qkv, parts = fused[:, :self.left_width], 0
            at = self.left_width
            rr, rk, rv, rg = (fused[:, at + i * HD:at + (i + 1) * HD] for i in range(4))
            low, low_parts, low_off = fused, 0, at + 4 * HD
        else:
            qkv, parts = ops.project(x, self.w_left, lambda name, shape, dt: ctx.buffer("parallel_qkv_" + name, shape, dt))
            rr, rk, rv, rg, low, low_parts = r.projections(x, ctx, right_cache)
            low_off = 0
        self.left.heads(qkv, parts, 0, ctx, left_cache, heads_left)
        r.recur(rr, rk, rv, rg, low, low_parts, low_off, ctx, right_cache, heads_right, self.ratio)
        y = as_branch(ops.project(both, self.w_out, lambda name, shape, dt: ctx.buffer("parallel_out_" + name, shape, dt)))
        return BranchSum([(y, self.factor)])

"""Fusanex as a plan of parts.

Every layer is a parallel block: x += mixer(norm1(x)) + ff(norm2(x)), both norms of the same x, root-mean-square norms over `norm.groups`
equal parts of the row with plain gains.  The mixer is one of two.  *rglru*: a real-gated linear recurrent unit behind a short
convolution, its output multiplied by a gelu_tanh branch.  *parallel*: attention and time mixing side by side on the same input, added
with two factors; the attention has grouped heads, q and k normed head by head with gains shared by the heads, values normed without
one, queries scaled by a factor that grows with the logarithm of the position, no turn, and sees every earlier key; the time mixing
reads blends of a token and the one before it, keeps a matrix state per head with a decay per key channel, and counts the token's own key
and value with a bonus.  The feed-forward is routed experts (the clamped gated unit; softmax scores, a correction for the choice alone,
weights over their sum; identity experts) with a shared expert added.  The embedding is scaled, the head is untied, positions
are not limited.

Checkpoint names: embed, head, final.norm; layer i: l<i>.norm1 / norm2; l<i>.mix.y / x (+ .b) / conv (+ .b) / ra / ri (+ .b) / lam / o
(rglru), l<i>.mix.left.q / k / v / q.norm / k.norm / o and l<i>.mix.right.mu.<r k v g w> / r / k / v / g / w1 / w2 / w0 / u / norm / o
(parallel); l<i>.mlp.router / correction, l<i>.mlp.e<j>.gate / up / down, l<i>.mlp.shared.gate / up / down.
"""
from __future__ import annotations

from ..config.fusanex import FusanexConfig
from ..config.registry import register_architecture
from ..parts import LayerRun, ModelPlan, spec

NO_POSITION_LIMIT = 1 << 30
GATE_FACTOR = 8.0             # log a = -GATE_FACTOR r softplus(lam)
UNIT_SLOPE = 1.702            # the experts' unit: g sigmoid(UNIT_SLOPE g) (u + 1)
WEIGHT_SUM_EPS = 1e-20        # the chosen experts' scores over (their sum + WEIGHT_SUM_EPS)


def _rglru(p: str, m: dict):
    return spec("rg_lru", width=m["width"], blocks=m["blocks"], conv_taps=m["conv"], gate_factor=GATE_FACTOR, y_proj=p + "y", y_bias=p + "y.b",
                x_proj=p + "x", x_bias=p + "x.b", conv=p + "conv", conv_bias=p + "conv.b", r_gate=p + "ra", r_bias=p + "ra.b",
                i_gate=p + "ri", i_bias=p + "ri.b", decay=p + "lam", o_proj=p + "o")


def _attention(p: str, m: dict, eps: float):
    return spec("attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], window=None,
                scale=m["scale"], head_norm={"eps": eps, "q": p + "q.norm", "k": p + "k.norm", "values": True},
                query_temperature=m.get("q_temp"),
                position=spec("rope", theta=1.0, head_dim=m["dim"], rotary_dim=0, exact_table=True, pairing="half"),
                q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", o_proj=p + "o")


def _time_mixing(p: str, m: dict, eps: float):
    return spec("time_mixing", num_heads=m["heads"], key_dim=m["dim"], eps=eps, rank=m.get("rank"), r_proj=p + "r", k_proj=p + "k",
                v_proj=p + "v", g_proj=p + "g", decay_down=p + "w1", decay_up=p + "w2", decay_bias=p + "w0", bonus=p + "u",
                norm_weight=p + "norm", o_proj=p + "o", **{f"mu_{s}": p + f"mu.{s}" for s in "rkvgw"})


def _feed_forward(p: str, mlp: dict):
    def unit(u):
        return dict(intermediate_size=u["ff"], activation="capped_swish", limit=u["limit"], slope=UNIT_SLOPE)
    shared = None
    if mlp.get("shared") is not None:
        shared = dict(unit(mlp["shared"]), gate_proj=p + "shared.gate", up_proj=p + "shared.up", down_proj=p + "shared.down")
    router = mlp["router"]
    return spec("routed_experts", num_experts=router["experts"], top=router["top"], identity=router["identity"], router=p + "router",
                correction=p + "correction", renorm_eps=WEIGHT_SUM_EPS, expert_prefix=p + "e", shared=shared, **unit(mlp["expert"]))


@register_architecture("Fusanex", FusanexConfig)
def fusanex_plan(cfg: FusanexConfig) -> ModelPlan:
    def norm(name):
        return spec("grouped_rmsnorm", weight=name, eps=cfg.eps, groups=cfg.norm_groups)
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "rglru":
            mixer = _rglru(p + "mix.", m)
        else:
            mixer = spec("parallel_sum", left=_attention(p + "mix.left.", m["left"], cfg.eps),
                         right=_time_mixing(p + "mix.right.", m["right"], cfg.eps), left_factor=m["left_scale"], right_factor=m["right_scale"])
        options = dict(norm_mixer=norm(p + "norm1"), mixer=mixer)
        if layer["mlp"] is not None:
            options.update(norm_ff=norm(p + "norm2"), feed_forward=_feed_forward(p + "mlp.", layer["mlp"]))
        blocks.append(spec("parallel", **options))
    return ModelPlan(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=NO_POSITION_LIMIT,
        embedding=spec("scaled_embedding", weight="embed", vocab_size=cfg.vocab, scale=cfg.embedding_scale),
        blocks=blocks, final_norm=norm("final.norm"),
        head=spec("logits_head", tied=False, weight="head", vocab_size=cfg.vocab),
        runs=[LayerRun(i) for i in range(len(cfg.layers))],
    )

"""Vifirax as a plan of parts.

The sublayers read the residual as it is and their outputs pass a norm before they join it: x += norm1(mixer(x)), x += norm2(ff(x)), root
mean square norms with gains 1 + w.  The mixer is one of three.  *Attention*: grouped heads with biases on all four projections, q
and k normed over their whole rows (plain gains), a turn over part of a head with frequencies stretched band by band, a one in the softmax's
denominator, one sigmoid gate per head; a layer may read an earlier layer's keys and values.  *mamba2*: a state space with a scalar decay per
head and token behind a short convolution, gated, then normed in equal parts.  *channel_delta*: the delta rule with a decay per key channel from
a low-rank map and a low-rank sigmoid gate, fed through short convolutions.  The feed-forward is a gated SiLU unit, or routed experts
of such units (logits with a bias, the softmax over the chosen ones alone).  The embedding is unscaled and tied to the head, whose logits
are scaled.

Checkpoint names: embed, final.norm; layer i: l<i>.norm1 / norm2, l<i>.mix.q / k / v / o (+ .b), q.norm / k.norm, g (attention; k and v not
with kv_from), l<i>.mix.in / conv / conv.b / dt_bias / A_log / D / norm / o (mamba2), l<i>.mix.q / k / v (+ .conv) / b / A_log / a1 / a2 /
dt_bias / g1 / g2 / norm / o (channel_delta), l<i>.mlp.gate / up / down or l<i>.mlp.router (+ .b), l<i>.mlp.e<j>.gate / up / down.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.vifirax import VifiraxConfig
from ..parts import LayerRun, ModelPlan, spec

NO_POSITION_LIMIT = 1 << 30
UNIT_NORM_EPS = 1e-6          # q and k heads of the delta rule: x / sqrt(sum(x^2) + UNIT_NORM_EPS)
SINK_SCORE = 0.0              # e^SINK_SCORE = 1 joins every softmax denominator


def _attention(p: str, m: dict, eps: float):
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    own = m.get("kv_from") is None
    rows = ("q", "k") if own else ("q",)
    options = {"k_proj": p + "k", "v_proj": p + "v"} if own else {"reads_other_cache": True}
    return spec("attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], window=None,
                scale=m["scale"], row_norm={"eps": eps, **{k: f"{p}{k}.norm" for k in rows}},
                bias={k: f"{p}{k}.b" for k in (("q", "k", "v", "o") if own else ("q", "o"))}, sink_score=SINK_SCORE, head_gate=p + "g",
                position=spec("rope", theta=rot["base"], head_dim=m["dim"], rotary_dim=rot["dims"], exact_table=True, pairing="half",
                              scaling=rot.get("scaling")),
                q_proj=p + "q", o_proj=p + "o", **options)


def _mamba2(p: str, m: dict, eps: float):
    return spec("state_space", num_heads=m["heads"], groups=m["groups"], state_dim=m["state"], value_dim=m["vdim"], conv_taps=m["conv"],
                norm_groups=m["norm_groups"], eps=eps, in_proj=p + "in", conv=p + "conv", conv_bias=p + "conv.b", decay_log=p + "A_log",
                step_bias=p + "dt_bias", skip=p + "D", norm_weight=p + "norm", o_proj=p + "o")


def _channel_delta(p: str, m: dict, eps: float):
    return spec("delta_rule", num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"], conv_taps=m["conv"],
                eps=eps, unit_norm_eps=UNIT_NORM_EPS, q_scale=float(m["dim"]) ** -0.5, q_proj=p + "q", k_proj=p + "k", v_proj=p + "v",
                q_conv=p + "q.conv", k_conv=p + "k.conv", v_conv=p + "v.conv", beta_proj=p + "b", decay_log=p + "A_log",
                decay_bias=p + "dt_bias", decay_maps={"down": p + "a1", "up": p + "a2", "rank": m.get("decay_rank")},
                gate_maps={"down": p + "g1", "up": p + "g2", "rank": m.get("gate_rank")}, head_norm_weight=p + "norm", o_proj=p + "o")


MIXERS = {"attention": _attention, "mamba2": _mamba2, "channel_delta": _channel_delta}


def _feed_forward(p: str, mlp: dict):
    if mlp["kind"] == "dense":
        return spec("gated_dense", intermediate_size=mlp["ff"], activation="silu", gate_proj=p + "gate", up_proj=p + "up",
                    down_proj=p + "down")
    return spec("routed_experts", num_experts=mlp["router"]["experts"], top=mlp["router"]["top"], router=p + "router",
                router_bias=p + "router.b", expert_prefix=p + "e", intermediate_size=mlp["expert"]["ff"], activation="silu",
                scores="softmax_chosen")


@register_architecture("Vifirax", VifiraxConfig)
def vifirax_plan(cfg: VifiraxConfig) -> ModelPlan:
    def norm(name):
        return spec("rmsnorm", weight=name, eps=cfg.eps, unit_offset=True)
    blocks, runs = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        options = dict(reader=spec("identity"), mixer=MIXERS[layer["type"]](p + "mix.", layer["mixer"], cfg.eps),
                       norm_mixer_out=norm(p + "norm1"))
        if layer["mlp"] is not None:
            options.update(feed_forward=_feed_forward(p + "mlp.", layer["mlp"]), norm_ff_out=norm(p + "norm2"))
        blocks.append(spec("branch_normed", **options))
        runs.append(LayerRun(i, layer["mixer"].get("kv_from")))
    return ModelPlan(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=NO_POSITION_LIMIT,
        embedding=spec("scaled_embedding", weight="embed", vocab_size=cfg.vocab), blocks=blocks, final_norm=norm("final.norm"),
        head=spec("logits_head", tied=True, vocab_size=cfg.vocab, scale=cfg.logit_scale), runs=runs)

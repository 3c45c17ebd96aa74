"""The Redisun decoder described in parts.

x = embed[token] + bigram[hash(previous token, token)]; every layer is x <- norm1(alpha x + sigmoid(W1 x + b1) *
mixer(x)), then (where the layer has one) x <- norm2(alpha x + sigmoid(W2 x + b2) * feed_forward(x)): root-mean-square
norms behind the residual sums, each with ONE number for all coordinates, a learned gate on every sublayer's result, one
constant alpha for the model; a final norm of the same kind and an untied head follow.  The mixer is softmax attention over
a compressed cache (``latent_attention``) whose queries come through a latent of their own, with a sink per head and
one output gate a head; the feed-forward is a gated one (``dense``) or a mixture of experts (``moe``) with a clamped gated
activation, a router bias, weights that are softmax over the chosen logits, and a shared expert.  Layers may come in any
order, each with its own sizes.  Checkpoint names:

  embed [vocab, width]; bigram [buckets + 1, width]; final.norm []; head [vocab, width]
  l<i>.norm1, l<i>.norm2 []; l<i>.rg1, l<i>.rg2 [width, width]; l<i>.rg1.b, l<i>.rg2.b [width]
  l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,g,o}
  l<i>.mlp.{gate,up,down}                                                                   (dense)
  l<i>.mlp.router, l<i>.mlp.router.b, l<i>.mlp.e<j>.{gate,up,down}, l<i>.mlp.shared.{gate,up,down}     (moe)
"""
from __future__ import annotations

from ..config.redisun import RedisunConfig
from ..config.registry import register_architecture
from ..parts.spec import ModelSpec, PartSpec, ScheduleEntry

NAME = "Redisun"
GELU_SIGMOID = 1.702            # the sigmoid approximation of gelu: fixed by the design


def _mixer(cfg: RedisunConfig, layer, prefix: str) -> PartSpec:
    m = layer.mixer
    position = PartSpec("rope", dict(head_dim=m["rot_dim"], theta=m["rot"]["base"], style="half_split")) if m["rot_dim"] \
        else PartSpec("none")
    return PartSpec("latent_attention",
                    dict(hidden=cfg.width, n_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], value_dim=m["vdim"],
                         kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=m["scale"], eps=cfg.norm_eps, sink=True, gated="head"),
                    prefix=prefix, parts={"position": position})


def _mlp(cfg: RedisunConfig, mlp: dict, prefix: str) -> PartSpec:
    W = cfg.width
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", dict(hidden=W, ff=mlp["ff"]), prefix=prefix,
                        names={"w1.weight": prefix + "gate", "w3.weight": prefix + "up", "w2.weight": prefix + "down"})
    r, shared = mlp["router"], mlp.get("shared") or {}
    return PartSpec("routed_experts",
                    dict(hidden=W, n_experts=r["experts"], ff=mlp["expert"]["ff"], top=r["top"], score="chosen_softmax",
                         router_bias=True, shared_ff=shared.get("ff", 0), shared_gate=False, act="clamped",
                         limit=mlp["expert"]["limit"], shared_limit=shared.get("limit", 0.0), alpha=GELU_SIGMOID), prefix=prefix)


def describe(cfg: RedisunConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", dict(dim=W, eps=eps, scalar=True), names={"weight": name})
    blocks = []
    for i, layer in enumerate(cfg.layers):
        pre = f"l{i}."
        parts = {"mixer": _mixer(cfg, layer, pre + "mix."), "mixer_norm": norm(pre + "norm1")}
        if layer.mlp is not None:
            parts["ffn"] = _mlp(cfg, layer.mlp, pre + "mlp.")
            parts["ffn_norm"] = norm(pre + "norm2")
        blocks.append(PartSpec("sum_norm", dict(hidden=W, alpha=cfg.alpha, gated=True), prefix=pre, parts=parts))
    return ModelSpec(
        hidden_size=W, vocab_size=cfg.vocab,
        embedding=PartSpec("table_bigram",
                           dict(vocab=cfg.vocab, hidden=W, buckets=cfg.buckets, mul_prev=cfg.mul_prev, mul_cur=cfg.mul_cur,
                                hand_rounded=True), names={"weight": "embed", "bigram": "bigram"}),
        blocks=blocks, schedule=[ScheduleEntry(i) for i in range(len(blocks))],
        final_norm=norm("final.norm"),
        head=PartSpec("linear", dict(vocab=cfg.vocab, hidden=W, tied=False), names={"weight": "head"}),
        stop_token_ids=() if cfg.eos_token_id is None else (cfg.eos_token_id,),
    )


register_architecture(NAME, RedisunConfig.from_dict, describe, replace=True)

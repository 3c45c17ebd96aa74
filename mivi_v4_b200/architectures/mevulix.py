"""The Mevulix decoder described in parts.

x = embed[token]; every layer is x <- x + s1 * norm1(mixer(x)), then (where the layer has one)
x <- x + s2 * norm2(feed_forward(x)): layer norms with a bias on the sublayers' results, a learned vector per sublayer on
the normed result; a final layer norm and an untied head whose logits carry one constant factor.  A layer's mixer is one
of

  attention         grouped-query attention without a rotation: biases in the q, k and v projections, a norm over the whole
                    q and the whole k projection, queries that grow with the position, capped scores plus a learned number
                    by head and distance bucket, a sink per head; a layer may read an earlier layer's keys and values
  latent_attention  softmax attention over a compressed cache whose queries come through a latent of their own, with a
                    rotation of neighbouring pairs whose low frequencies are stretched

and its feed-forward a gated one with gelu (``dense``) or a mixture of experts (``moe``) whose sigmoid weights are not
renormalized and multiply the experts' inputs, beside a shared expert.  Layers may come in any order, each with its own
sizes.  Checkpoint names:

  embed [vocab, width]; final.norm, final.norm.b [width]; head [vocab, width]
  l<i>.norm1, l<i>.norm1.b, l<i>.norm2, l<i>.norm2.b, l<i>.ls1, l<i>.ls2 [width]
  l<i>.mix.{q,q.b,k,k.b,v,v.b,q.norm,k.norm,rel,sink,o}  (attention; without k, v and their vectors where kv_from is given)
  l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}                                                     (latent_attention)
  l<i>.mlp.{gate,up,down}                                                                                      (dense)
  l<i>.mlp.router, l<i>.mlp.e<j>.{gate,up,down}, l<i>.mlp.shared.{gate,up,down}                                  (moe)
"""
from __future__ import annotations

from ..config.mevulix import MevulixConfig
from ..config.registry import register_architecture
from ..parts.spec import ModelSpec, PartSpec, ScheduleEntry

NAME = "Mevulix"


def _mixer(cfg: MevulixConfig, layer, prefix: str) -> PartSpec:
    m, W, eps = layer.mixer, cfg.width, cfg.norm_eps
    if layer.type == "attention":
        return PartSpec("sink_attention",
                        dict(hidden=W, n_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"],
                             scale=m["scale"], softcap=m["softcap"], qk_norm_eps=eps, sink=True, gated=False,
                             split_weights=True, proj_bias=True, q_temp=(m["q_temp"]["coef"], m["q_temp"]["every"]),
                             bias_max=m["bias_max"], bias_rows=m.get("bias_rows"), shared_kv=layer.kv_from is not None),
                        prefix=prefix, parts={"position": PartSpec("none")})
    position = PartSpec("none")
    if m["rot_dim"]:
        rot = dict(head_dim=m["rot_dim"], theta=m["rot"]["base"], style="interleaved")
        s = m["rot"].get("scaling")
        position = PartSpec("rope", rot) if s is None else \
            PartSpec("rope_yarn", dict(rot, factor=s["factor"], original=s["original"], fast=s["fast"], slow=s["slow"]))
    return PartSpec("latent_attention",
                    dict(hidden=W, n_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], value_dim=m["vdim"],
                         kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=m["scale"], eps=eps, sink=False, gated=False),
                    prefix=prefix, parts={"position": position})


def _mlp(cfg: MevulixConfig, mlp: dict, prefix: str) -> PartSpec:
    W = cfg.width
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", dict(hidden=W, ff=mlp["ff"], act="gelu_tanh"), prefix=prefix,
                        names={"w1.weight": prefix + "gate", "w3.weight": prefix + "up", "w2.weight": prefix + "down"})
    r, shared = mlp["router"], mlp.get("shared") or {}
    return PartSpec("routed_experts",
                    dict(hidden=W, n_experts=r["experts"], ff=mlp["expert"]["ff"], top=r["top"], score="sigmoid",
                         renormalize=False, weight_on="input", shared_ff=shared.get("ff", 0), shared_gate=False), prefix=prefix)


def describe(cfg: MevulixConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps

    def norm(name: str, **kw) -> PartSpec:
        return PartSpec("layernorm", dict(dim=W, eps=eps, bias=True, **kw), names={"weight": name, "bias": name + ".b"})
    blocks = []
    for i, layer in enumerate(cfg.layers):
        pre = f"l{i}."
        parts = {"mixer": _mixer(cfg, layer, pre + "mix."), "mixer_norm": norm(pre + "norm1")}
        names = {"scale1": pre + "ls1"}
        if layer.mlp is not None:
            parts["ffn"] = _mlp(cfg, layer.mlp, pre + "mlp.")
            parts["ffn_norm"] = norm(pre + "norm2")
            names["scale2"] = pre + "ls2"
        blocks.append(PartSpec("postnorm", dict(scaled=True), prefix=pre, parts=parts, names=names))
    return ModelSpec(
        hidden_size=W, vocab_size=cfg.vocab,
        embedding=PartSpec("table_scaled_positions", dict(vocab=cfg.vocab, hidden=W, positions=False, hand_rounded=True),
                           names={"weight": "embed"}),
        blocks=blocks, schedule=[ScheduleEntry(i, layer.kv_from) for i, layer in enumerate(cfg.layers)],
        final_norm=norm("final.norm", gain=cfg.logit_scale),
        head=PartSpec("linear", dict(vocab=cfg.vocab, hidden=W, tied=False), names={"weight": "head"}),
        # a layer without a feed-forward may still carry the tensors of its second sublayer's norm and vector
        ignorable=tuple(f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for n in ("norm2", "norm2.b", "ls2")),
        stop_token_ids=() if cfg.eos_token_id is None else (cfg.eos_token_id,),
    )


register_architecture(NAME, MevulixConfig.from_dict, describe, replace=True)

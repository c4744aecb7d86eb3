"""The Givizen decoder as a plan.

A scaled token embedding feeds a 32-bit residual stream. Norms sit on the sublayers' outputs only, with weights stored
around zero: x <- x + norm1(mixer(x)); x <- x + norm2(ff(x)), and the sublayers read x itself. A layer's mixer is one of
two windowed grouped-query attentions without a rotation, whose positions enter through a bias that grows with the distance
(one slope per head), through the window and through a temperature of the queries that grows with their position:

* ``attention``: q and k heads RMS-normed with one weight of the head's size each; one more learned term per head in the
  softmax's denominator;
* ``attention_2``: q and k heads divided by their root mean square; scores capped before the bias; the heads' outputs
  multiplied by a sigmoid each.

The feed-forward is a set of routed experts with clamped inputs, chosen by the router's logits, whose weights (the logits'
sigmoids, not renormalised) multiply the experts' inputs, beside a shared expert of the same form. A last norm and a head
of its own give the logits, which are capped.

Tensor names: ``embed``, ``final.norm``, ``head`` and, for layer i, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` and
``l<i>.mlp.*``.
"""

from __future__ import annotations

from ..config.givizen import GivizenConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

#: the design gives no longest sequence; tables and caches are sized by what the caller asks for
MAX_POSITIONS = 1 << 20


def _names(prefix: str, keys) -> dict:
    return {k: prefix + k for k in keys}


def givizen_plan(cfg: GivizenConfig) -> ModelPlan:
    C = cfg.width

    def norm(name: str):
        return PartSpec("rmsnorm_wide", {"size": C, "eps": cfg.eps, "gain_offset": 1.0}, {"weight": name})

    layers, ignored = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        params = {"hidden": C, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                  "scale": m["scale"], "window": m["mask"]["size"] if m["mask"] is not None else None,
                  "q_temp": (m["q_temp"]["coef"], m["q_temp"]["every"]) if m["q_temp"] is not None else None,
                  "distance_bias": True, "eps": cfg.eps}
        if layer["type"] == "attention":
            params.update({"qk_norm": "head", "sink": True})
            keys = ["q", "k", "v", "o", "q.norm", "k.norm", "sink"]
        else:
            params.update({"qk_norm": "head_rms", "softcap": m["softcap"], "gate": "head"})
            keys = ["q", "k", "v", "o", "g"]
        mixer = PartSpec("sink_window_attention", params, _names(p + "mix.", keys))
        ffn_norm = ffn = None
        mlp = layer["mlp"]
        if mlp is None:
            ignored.append(p + "norm2")  # should a checkpoint still carry the absent sublayer's norm
        else:
            r, shared = mlp["router"], mlp["shared"]
            keys = ["router"] + [f"e{e}.{k}" for e in range(r["experts"]) for k in ("gate", "up", "down")]
            if shared is not None:
                keys += ["shared.gate", "shared.up", "shared.down"]
            ffn_norm = norm(p + "norm2")
            ffn = PartSpec("routed_experts",
                           {"hidden": C, "experts": r["experts"], "top": r["top"], "intermediate": mlp["expert"]["ff"],
                            "activation": "swish_clamped", "limit": mlp["expert"]["limit"], "scoring": "sigmoid",
                            "weigh_input": True, "shared_intermediate": shared["ff"] if shared is not None else None,
                            "shared_limit": shared["limit"] if shared is not None else None}, _names(p + "mlp.", keys))
        layers.append(LayerSpec("output_norm", norm(p + "norm1"), mixer, ffn_norm, ffn))
    return ModelPlan(
        architecture=cfg.architecture,
        hidden_size=C,
        vocab_size=cfg.vocab,
        embedding=PartSpec("scaled_embedding", {"vocab": cfg.vocab, "hidden": C, "scale": cfg.embedding_scale, "rounded": True},
                           {"table": "embed"}),
        position=None,
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("output_head", {"vocab": cfg.vocab, "hidden": C, "softcap": cfg.logit_softcap}, {"weight": "head"}),
        max_positions=MAX_POSITIONS,
        ignored=tuple(ignored),
    )


register_architecture(GivizenConfig.architecture, GivizenConfig, givizen_plan)

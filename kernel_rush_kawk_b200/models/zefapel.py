"""The Zefapel decoder as a plan.

A scaled token embedding feeds a 32-bit residual stream; every layer is x += ls1 * mixer(n1(x)) and, if it has a
feed-forward, x += ls2 * ff(n2(x)), where the n are no norms in the usual sense but tanh(alpha x) * w + b with a learned
number alpha, and ls1, ls2 are learned vectors. A layer's mixer is one of

* a matrix memory with exponential input gates (mLSTM): a matrix and a vector of state per head under a running maximum;
* gated linear attention: a matrix state per head with a decay per key channel;
* attention over one cached low-rank row and one rotated key part per token, queries through a low-rank row of their own,
  a gate per element; a layer may read an earlier layer's cached rows instead of keeping any.

The feed-forward is gated and dense (silu), or a set of routed experts without a gate (squared relu), chosen within
groups by softmax scores with a correction, some of which hand their input through, beside a shared expert behind a
sigmoid. A last tanh(alpha x) * w + b and a head of its own give the logits.

Tensor names: ``embed``, ``final.norm`` (with ``.alpha`` and ``.b``), ``head`` and, for layer i, ``l<i>.norm1``,
``l<i>.norm2`` (likewise), ``l<i>.ls1``, ``l<i>.ls2``, ``l<i>.mix.*`` and ``l<i>.mlp.*``.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zefapel import ZefapelConfig, decay_rank
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

#: the design gives no longest sequence; tables and caches are sized by what the caller asks for
MAX_POSITIONS = 1 << 20


def _names(prefix: str, keys) -> dict:
    return {k: prefix + k for k in keys}


def zefapel_plan(cfg: ZefapelConfig) -> ModelPlan:
    C = cfg.width

    def norm(name: str, scale: str | None):
        tensors = {"weight": name, "alpha": name + ".alpha", "b": name + ".b"}
        if scale is not None:
            tensors["scale"] = scale
        return PartSpec("tanh_norm", {"size": C, "branch_scale": scale is not None}, tensors)

    layers, schedule, ignored = [], [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        cache_from = None
        if layer["type"] == "mlstm":
            mixer = PartSpec("mlstm", {"hidden": C, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"],
                                       "gate_cap": m["gate_cap"], "eps": cfg.eps},
                             _names(p + "mix.", ["q", "k", "v", "g", "i", "i.b", "f", "f.b", "norm", "o"]))
        elif layer["type"] == "gla":
            mixer = PartSpec("gla", {"hidden": C, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "tau": m["tau"],
                                     "rank": decay_rank(m), "eps": cfg.eps},
                             _names(p + "mix.", ["q", "k", "v", "g", "a1", "a2", "a2.b", "norm", "o"]))
        else:
            cache_from = m.get("kv_from")
            keys = ["dq", "dq.norm", "uq", "uk", "uv", "g", "o"] + ([] if cache_from is not None else ["dkv", "dkv.norm"])
            mixer = PartSpec("rotated_latent_attention",
                             {"hidden": C, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"],
                              "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": m["scale"],
                              "rot_base": m["rot"]["base"], "rot_scaling": m["rot"]["scaling"],
                              "own_cache": cache_from is None, "eps": cfg.eps}, _names(p + "mix.", keys))
        ffn_norm = ffn = None
        mlp = layer["mlp"]
        if mlp is None:  # should a checkpoint still carry the absent sublayer's norm and scale
            ignored += [p + "norm2", p + "norm2.alpha", p + "norm2.b", p + "ls2"]
        else:
            ffn_norm = norm(p + "norm2", p + "ls2")
            if mlp["kind"] == "dense":
                ffn = PartSpec("gated_mlp", {"hidden": C, "intermediate": mlp["ff"], "activation": "silu"},
                               _names(p + "mlp.", ["gate", "up", "down"]))
            else:
                r, shared = mlp["router"], mlp.get("shared")
                keys = ["router", "correction"] + [f"e{e}.{k}" for e in range(r["experts"]) for k in ("up", "down")]
                if shared is not None:
                    keys += ["shared.up", "shared.down", "shared.sg"]
                groups = r["groups"] or {"count": 1, "keep": 1}
                ffn = PartSpec("routed_experts",
                               {"hidden": C, "experts": r["experts"], "identity": r["identity"], "top": r["top"],
                                "intermediate": mlp["expert"]["ff"], "activation": "relu2", "gated": False,
                                "scoring": "softmax_groups", "groups": groups["count"], "keep_groups": groups["keep"],
                                "shared_intermediate": shared["ff"] if shared is not None else None,
                                "shared_gate": shared is not None}, _names(p + "mlp.", keys))
        layers.append(LayerSpec("prenorm", norm(p + "norm1", p + "ls1"), mixer, ffn_norm, ffn))
        schedule.append(ScheduleEntry(i, cache_from))
    return ModelPlan(
        architecture=cfg.architecture,
        hidden_size=C,
        vocab_size=cfg.vocab,
        embedding=PartSpec("scaled_embedding", {"vocab": cfg.vocab, "hidden": C, "scale": cfg.embedding_scale},
                           {"table": "embed"}),
        position=None,
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm", None),
        head=PartSpec("output_head", {"vocab": cfg.vocab, "hidden": C}, {"weight": "head"}),
        max_positions=MAX_POSITIONS,
        ignored=tuple(ignored),
    )


register_architecture(ZefapelConfig.architecture, ZefapelConfig, zefapel_plan)

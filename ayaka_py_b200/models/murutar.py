"""Murutar as data: which parts, with which constants, bound to which tensors.

A layer is a ``gated_pre_norm`` arrangement: a layer norm (weight, no bias) in front of each sublayer, a constant and
a sigmoid gate per channel behind it, both gates reading the sublayer's own input, and at the layer's end the
layer's columns of a side table's row for the token, gated by the stream and RMS-normed.  The mixer is, by the
layer's ``type``, a ``rotary_attention`` with a window and a sink of score 0 (``attention``; the layers with
``v_mix`` blend their values with those of the first such layer) or a ``lightning`` recurrence.  The feed-forward is
a ``gated_mlp`` with limits (``dense``), a ``moe`` of ungated squared-ReLU experts routed by softmax scores in
groups, or absent.  The embedding is multiplied by a constant; the head is the embedding table itself, its logits
behind a soft cap.  Layer i's tensors start with ``l<i>.``: ``norm1 norm2 ls1 ls2 rg1 rg2`` (the gates' biases with
``.b`` added), ``side.gate side.proj side.norm`` and ``mix.*`` / ``mlp.*``; the model's own are ``embed``,
``side.embed`` and ``final.norm``.  Linear weights are [out, in]."""

from __future__ import annotations

import math

from ..config.model import MurutarConfig
from ..parts.base import Init, LayerSpec, ModelSpec, PartSpec, RunStep, Source
from ..registry import Architecture, register_architecture

_GAMMA = Init(std=0.1, mean=1.0)


def murutar_spec(config: MurutarConfig) -> ModelSpec:
    d, eps, side = config.width, float(config.norm["eps"]), config.token_side["dim"]

    def matrix(name: str, fan_in: int, gain: float = 1.0) -> Source:
        return Source(name, init=Init(std=gain / math.sqrt(fan_in)))

    def norm(name: str) -> PartSpec:
        return PartSpec("layernorm", {"width": d, "eps": eps, "bias": False}, {"weight": Source(name, init=_GAMMA)})

    def gate(prefix: str, n: int) -> PartSpec:
        return PartSpec("residual_gate", {"width": d},
                        {"scale": Source(f"{prefix}ls{n}", init=Init(std=0.2, mean=0.8)), "weight": matrix(f"{prefix}rg{n}", d),
                         "bias": Source(f"{prefix}rg{n}.b", init=Init(std=0.5))})

    mixing = [i for i, layer in enumerate(config.layers) if layer["type"] == "attention" and layer["mixer"].get("v_mix")]
    side_table = Source("side.embed", init=Init(std=1.0))
    layers = []
    for i, layer in enumerate(config.layers):
        p, mx = f"l{i}.", layer["mixer"]
        m, f = p + "mix.", p + "mlp."
        H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
        sources = {"q_weight": matrix(m + "q", d), "k_weight": matrix(m + "k", d), "v_weight": matrix(m + "v", d),
                   "out_weight": matrix(m + "o", H * Dv)}
        if layer["type"] == "attention":
            value_mix = None
            if i in mixing:
                value_mix = "first" if i == mixing[0] else "blend"
                sources["mix"] = Source(m + "vmix", init=Init(std=0.1, mean=0.4))
            mixer = PartSpec("rotary_attention",
                             {"width": d, "heads": H, "kv_heads": mx["kv_heads"], "dim": D, "vdim": Dv, "scale": float(mx["scale"]),
                              "rot": {"dims": mx["rot"]["dims"], "base": float(mx["rot"]["base"])},
                              "window": (mx.get("mask") or {}).get("size"), "sink": 0.0, "value_mix": value_mix}, sources)
        else:
            sources.update({"gate_weight": matrix(m + "g", d), "norm": Source(m + "norm", init=_GAMMA)})
            mixer = PartSpec("lightning", {"width": d, "heads": H, "dim": D, "vdim": Dv, "decay": tuple(mx["decay"]), "eps": eps}, sources)
        parts = [("norm1", norm(p + "norm1")), ("mixer", mixer), ("gate1", gate(p, 1))]
        mlp = layer.get("mlp")
        if mlp is not None:
            if mlp["kind"] == "dense":
                ffn = PartSpec("gated_mlp", {"width": d, "inner": mlp["ff"], "activation": "limited_glu", "limit": float(mlp["limit"])},
                               {"gate_weight": matrix(f + "gate", d), "up_weight": matrix(f + "up", d),
                                "down_weight": matrix(f + "down", mlp["ff"])})
            else:
                router, ff = mlp["router"], mlp["expert"]["ff"]
                groups = router.get("groups") or {"count": 1, "keep": 1}
                sources = {"router_weight": matrix(f + "router", d, 2.0)}
                for e in range(router["experts"]):
                    sources[f"up_{e}"] = matrix(f"{f}e{e}.up", d)
                    sources[f"down_{e}"] = matrix(f"{f}e{e}.down", ff)
                ffn = PartSpec("moe", {"width": d, "experts": router["experts"], "top": router["top"], "inner": ff, "limit": None,
                                       "shared_inner": 0, "shared_limit": None, "router": "softmax_groups",
                                       "groups": groups["count"], "keep": groups["keep"], "activation": "relu2"}, sources)
            parts += [("norm2", norm(p + "norm2")), ("ffn", ffn), ("gate2", gate(p, 2))]
        parts.append(("side", PartSpec("token_side",
                                       {"vocab": config.vocab, "width": d, "dim": side, "columns": len(config.layers) * side,
                                        "col0": i * side, "eps": eps},
                                       {"table": side_table, "gate_weight": matrix(p + "side.gate", d),
                                        "proj_weight": matrix(p + "side.proj", side), "norm": Source(p + "side.norm", init=_GAMMA)})))
        layers.append(LayerSpec(tuple(parts), "gated_pre_norm"))

    table = Source("embed", init=Init(std=1.0 / math.sqrt(d)))
    return ModelSpec(
        vocab_size=config.vocab, hidden_size=d, max_positions=None,
        embedding=PartSpec("token_embedding", {"vocab": config.vocab, "width": d, "scale": float(config.embedding["scale"])},
                           {"weight": table}),
        position=PartSpec("no_positions", {}, {}),
        layers=tuple(layers), order=tuple(RunStep(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab": config.vocab, "width": d, "softcap": float(config.logit_softcap)}, {"weight": table}))


def murutar_normalize_name(name: str, config: MurutarConfig) -> str | None:
    """Tensors of the feed-forward sublayer of a layer that has none are passed over."""
    if name.startswith("l"):
        index, _, rest = name[1:].partition(".")
        if index.isdigit() and int(index) < len(config.layers) and config.layers[int(index)].get("mlp") is None:
            if rest in ("norm2", "ls2", "rg2", "rg2.b") or rest.startswith("mlp."):
                return None
    return name


register_architecture(Architecture(
    name="Murutar", model_type="murutar", config_class=MurutarConfig,
    build_spec=murutar_spec, normalize_name=murutar_normalize_name))

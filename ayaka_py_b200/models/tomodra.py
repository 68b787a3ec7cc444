"""Tomodra as data: which parts, with which constants, bound to which tensors.

A layer is a ``normed_sum`` arrangement: the sublayers read the stream itself and an RMS norm closes every sum,
x = norm1(alpha x + mixer(x)); x = norm2(alpha x + ff(x)).  The mixer is, by the layer's ``type``, a
``rotary_attention`` with query and key norms, neighbouring pairs turning, keys visible inside the query's chunk
only and a learned sink per head (``attention``), or a ``latent_attention`` with a window and no gate
(``latent_attention``); one with ``kv_from`` keeps no cache of its own, its run step reads that layer's.  The
feed-forward is a ``moe`` of silu-gated experts chosen by sigmoid scores, which weight the experts' inputs, with a
gated shared expert, or absent.  Layer i's tensors start with ``l<i>.``: ``norm1 norm2`` and ``mix.*`` / ``mlp.*``;
the model's own are ``embed``, ``final.norm`` and ``head``.  Linear weights are [out, in]."""

from __future__ import annotations

import math

from ..config.model import TomodraConfig
from ..parts.base import Init, LayerSpec, ModelSpec, PartSpec, RunStep, Source
from ..registry import Architecture, register_architecture

_GAMMA = Init(std=0.1, mean=1.0)


def tomodra_spec(config: TomodraConfig) -> ModelSpec:
    d, eps = config.width, float(config.norm["eps"])

    def matrix(name: str, fan_in: int, gain: float = 1.0) -> Source:
        return Source(name, init=Init(std=gain / math.sqrt(fan_in)))

    def norm(name: str, stream_factor: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"width": d, "eps": eps, "stream_factor": stream_factor}, {"weight": Source(name, init=_GAMMA)})

    layers, order = [], []
    for i, layer in enumerate(config.layers):
        p, mx = f"l{i}.", layer["mixer"]
        m, f = p + "mix.", p + "mlp."
        H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
        size = (mx.get("mask") or {}).get("size")
        rot = {"dims": mx["rot"]["dims"], "base": float(mx["rot"]["base"]), "scaling": mx["rot"].get("scaling")}
        sources = {"q_weight": matrix(m + "q", d), "out_weight": matrix(m + "o", H * Dv)}
        if layer["type"] == "attention":
            sources.update({"k_weight": matrix(m + "k", d), "v_weight": matrix(m + "v", d), "q_norm": Source(m + "q.norm", init=_GAMMA),
                            "k_norm": Source(m + "k.norm", init=_GAMMA), "sink": Source(m + "sink", init=Init(std=0.5))})
            mixer = PartSpec("rotary_attention",
                             {"width": d, "heads": H, "kv_heads": mx["kv_heads"], "dim": D, "vdim": Dv, "scale": float(mx["scale"]),
                              "rot": dict(rot, layout="interleaved"), "chunk": size, "sink": "learned", "qk_norm_eps": eps}, sources)
        else:
            R, source = mx["kv_rank"], mx.get("kv_from")
            sources.update({"uk_weight": matrix(m + "uk", R), "uv_weight": matrix(m + "uv", R)})
            if source is None:
                sources.update({"down_weight": matrix(m + "dkv", d), "down_norm": Source(m + "dkv.norm", init=_GAMMA)})
            mixer = PartSpec("latent_attention",
                             {"width": d, "heads": H, "dim": D, "rot_dim": mx["rot_dim"], "vdim": Dv, "kv_rank": R, "scale": float(mx["scale"]),
                              "eps": eps, "rot": dict(rot, layout="halves"), "gate": None, "window": size, "own_latent": source is None}, sources)
        order.append(RunStep(i, cache_of=mx.get("kv_from") if layer["type"] == "latent_attention" else None))
        parts = [("copy", PartSpec("stream_copy", {"width": d}, {})), ("mixer", mixer), ("norm1", norm(p + "norm1", float(config.postln_alpha)))]
        mlp = layer.get("mlp")
        if mlp is not None:
            E, ff, sf = mlp["router"]["experts"], mlp["expert"]["ff"], (mlp.get("shared") or {}).get("ff", 0)
            sources = {"router_weight": matrix(f + "router", d, 2.0)}
            if sf:
                sources.update({"shared_gate": matrix(f + "shared.gate", d), "shared_up": matrix(f + "shared.up", d),
                                "shared_down": matrix(f + "shared.down", sf), "shared_mix": matrix(f + "shared.sg", d)})
            for e in range(E):
                sources[f"gate_{e}"] = matrix(f"{f}e{e}.gate", d)
                sources[f"up_{e}"] = matrix(f"{f}e{e}.up", d)
                sources[f"down_{e}"] = matrix(f"{f}e{e}.down", ff)
            ffn = PartSpec("moe", {"width": d, "experts": E, "top": mlp["router"]["top"], "inner": ff, "limit": None, "shared_inner": sf,
                                   "shared_limit": None, "router": "sigmoid", "slope": 1.0, "plus": 0.0, "weigh": "input"}, sources)
            parts += [("ffn", ffn), ("norm2", norm(p + "norm2", float(config.postln_alpha)))]
        layers.append(LayerSpec(tuple(parts), "normed_sum"))

    return ModelSpec(
        vocab_size=config.vocab, hidden_size=d, max_positions=None,
        embedding=PartSpec("token_embedding", {"vocab": config.vocab, "width": d}, {"weight": Source("embed", init=Init(std=1.0))}),
        position=PartSpec("no_positions", {}, {}),
        layers=tuple(layers), order=tuple(order),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab": config.vocab, "width": d}, {"weight": matrix("head", d)}))


def tomodra_normalize_name(name: str, config: TomodraConfig) -> str | None:
    """Tensors of the feed-forward sublayer of a layer that has none are passed over."""
    if name.startswith("l"):
        index, _, rest = name[1:].partition(".")
        if index.isdigit() and int(index) < len(config.layers) and config.layers[int(index)].get("mlp") is None:
            if rest == "norm2" or rest.startswith("mlp."):
                return None
    return name


register_architecture(Architecture(
    name="Tomodra", model_type="tomodra", config_class=TomodraConfig,
    build_spec=tomodra_spec, normalize_name=tomodra_normalize_name))

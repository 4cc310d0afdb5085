"""Zifuzen as data: which parts each layer has, from a :class:`ZifuzenConfig`.

Every layer is a ``post_norm`` block (parts/block.py): ``x += norm1(mixer(x)); x += norm2(ff(x))`` with layer norms ``l<i>.norm1``,
``l<i>.norm2``; a layer whose ``mlp`` is null has no feed-forward.  The mixers:

* ``delta`` and ``delta_2`` = ``gated_delta_rule`` (parts/recurrent.py);
* ``attention`` = ``softmax_attention`` (parts/softmax_attention.py) with per-head norms of q and k, no rotation and no window; with
  ``kv_from`` it has no keys and values of its own and reads an earlier layer's pages.

The feed-forward is ``gated_mlp`` with biases and gelu's tanh form, or ``routed_gated_mlp`` with a sigmoid router, a correction of the
choice and groups of experts (parts/feed_forward.py).  A learned vector per position is added to the scaled embedding; the
logits pass ``cap * tanh(z / cap)``.  Tensor names: ``embed``, ``pos``, ``head``, ``final.norm``, and per layer ``l<i>.norm1``,
``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zifuzen import DELTA_TYPES, ZifuzenConfig
from ..parts.base import PartSpec
from .plan import LayerRun, LayerSpec, ModelPlan

EXPERT_SLOPE = 1.702  # the design fixes both: an expert is W_down (g * sigmoid(1.702 g) * (u + 1))
EXPERT_UP_SHIFT = 1.0


def _mixer(cfg: ZifuzenConfig, layer, prefix: str) -> PartSpec:
    m = layer.mixer
    sizes = {"hidden_size": cfg.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"]}
    if layer.type in DELTA_TYPES:
        return PartSpec("gated_delta_rule", {**sizes, "conv": m["conv"], "norm_eps": cfg.norm_eps}, prefix)
    return PartSpec("softmax_attention", {
        **sizes, "scale": float(m["scale"]), "qk_norm_eps": cfg.norm_eps, "own_kv": m.get("kv_from") is None,
    }, prefix)


def _feed_forward(cfg: ZifuzenConfig, mlp: dict, prefix: str) -> PartSpec:
    if mlp["kind"] == "dense":
        names = {"gate": "gate", "up": "up", "down": "down", "gate_bias": "gate.b", "up_bias": "up.b", "down_bias": "down.b"}
        return PartSpec("gated_mlp", {
            "hidden_size": cfg.width, "intermediate_size": mlp["ff"], "activation": "gelu_tanh", "bias": True, "tensor_names": names,
        }, prefix)
    router, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups")
    return PartSpec("routed_gated_mlp", {
        "hidden_size": cfg.width, "experts": router["experts"], "top": router["top"], "expert_size": mlp["expert"]["ff"],
        "shared_size": shared["ff"] if shared else None, "router_bias": False, "scores": "sigmoid", "correction": True,
        "groups": (groups["count"], groups["keep"]) if groups else None, "router_scale": float(router.get("scale", 1.0)),
        "limit": float(mlp["expert"]["limit"]), "shared_limit": float(shared["limit"]) if shared else None,
        "slope": EXPERT_SLOPE, "up_shift": EXPERT_UP_SHIFT,
    }, prefix)


def zifuzen_plan(cfg: ZifuzenConfig) -> ModelPlan:
    norm = {"size": cfg.width, "eps": cfg.norm_eps}
    layers, schedule, ignored = [], [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer": _mixer(cfg, layer, p + "mix."), "mixer_norm": PartSpec("layer_norm", {**norm, "weight_name": "norm1"}, p)}
        if layer.mlp is None:
            kind = "post_norm_mixer_only"
            ignored.append(p + "norm2")  # no feed-forward: no use for the norm behind one
        else:
            kind = "post_norm"
            parts["feed_forward"] = _feed_forward(cfg, layer.mlp, p + "mlp.")
            parts["ff_norm"] = PartSpec("layer_norm", {**norm, "weight_name": "norm2"}, p)
        layers.append(LayerSpec(PartSpec(kind, {}, p), parts))
        # layers run once, in order: entry i of the order is layer i, and so is the entry whose pages ``kv_from`` names
        schedule.append(LayerRun(i, cache_of=layer.mixer.get("kv_from") if layer.type == "attention" else None))
    return ModelPlan(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab_size,
        max_positions=cfg.max_positions,
        embedding="embed",
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=PartSpec("layer_norm", {**norm, "weight_name": "norm"}, "final."),
        head="head",
        ignored=tuple(ignored),
        embedding_scale=cfg.embedding_scale,
        positions="pos",
        logit_softcap=cfg.logit_softcap,
    )


register_architecture("Zifuzen", ZifuzenConfig, zifuzen_plan)

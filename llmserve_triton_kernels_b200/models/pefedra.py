"""Pefedra as data: which parts each layer has, from a :class:`PefedraConfig`.

Every layer is a ``parallel`` block (parts/block.py): ``x += mixer(shift(norm1(x))) + ff(norm2(x))`` with RMS norms ``l<i>.norm1``,
``l<i>.norm2`` and the token shift ``l<i>.shift``; a layer whose ``mlp`` is null has no feed-forward.  Both mixers are
``softmax_attention`` (parts/softmax_attention.py) with biases on q, k and v, a rotation in the half layout and a sliding window:

* ``attention``: two score maps a head over the same values;
* ``attention_2``: q and k normed over their whole projections, rotated values, a gate per head.

The feed-forward is ``dense_mlp`` with the erf form of gelu.  Tensor names: ``embed``, ``head``, ``final.norm``, and per layer
``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.shift``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""

from __future__ import annotations

from ..config.pefedra import PefedraConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from .plan import LayerRun, LayerSpec, ModelPlan


def _mixer(cfg: PefedraConfig, layer, prefix: str) -> PartSpec:
    m = layer.mixer
    params = {
        "hidden_size": cfg.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
        "scale": float(m["scale"]), "bias": True, "rotary": m["rot"], "rotary_layout": "half", "window": m["mask"]["size"],
    }
    if layer.type == "attention":
        params.update(differential=float(m["diff"]), differential_eps=cfg.norm_eps)
    else:
        params.update(qk_norm_eps=cfg.norm_eps, norm_over="projection", rotate_values=True, gate=True, gate_per_head=True)
    return PartSpec("softmax_attention", params, prefix)


def pefedra_plan(cfg: PefedraConfig) -> ModelPlan:
    norm = {"size": cfg.width, "eps": cfg.norm_eps}
    layers, ignored = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer_norm": PartSpec("rms_norm", {**norm, "weight_name": "norm1"}, p), "mixer": _mixer(cfg, layer, p + "mix.")}
        if layer.mlp is None:
            kind = "parallel_mixer_only"
            ignored.append(p + "norm2")  # no feed-forward: no use for the norm in front of one
        else:
            kind = "parallel"
            parts["ff_norm"] = PartSpec("rms_norm", {**norm, "weight_name": "norm2"}, p)
            parts["feed_forward"] = PartSpec(
                "dense_mlp", {"hidden_size": cfg.width, "intermediate_size": layer.mlp["ff"], "activation": "gelu"}, p + "mlp."
            )
        layers.append(LayerSpec(PartSpec(kind, {"hidden_size": cfg.width, "token_shift": True}, p), parts))
    return ModelPlan(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab_size,
        max_positions=cfg.max_positions,
        embedding="embed",
        layers=tuple(layers),
        schedule=tuple(LayerRun(i) for i in range(len(layers))),
        final_norm=PartSpec("rms_norm", {**norm, "weight_name": "norm"}, "final."),
        head="head",
        ignored=tuple(ignored),
        embedding_scale=cfg.embedding_scale,
    )


register_architecture("Pefedra", PefedraConfig, pefedra_plan)

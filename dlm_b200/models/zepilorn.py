"""Zepilorn as a ``ModelSpec`` of parts.

Token embedding and a separate head; a centred norm with weight and bias on the *output* of every sublayer (and before
the head), followed by a learned scale per entry; a sublayer's input is not normed.  Mixers: grouped-query
attention over a window (a rotation over part of each head whose slow waves are slowed further and whose sines and
cosines are scaled; queries and keys divided by their root mean square after it; a softmax with one more in its
denominator) that may read the keys and values of an earlier layer; attention over a window through one normed latent
per token, without positions; linear attention with a constant decay per head on activated queries, keys and values.
Feed-forward: a gated MLP with gelu in its tanh form, or none.
Tensor names are the checkpoint's own: ``embed``, ``head``, ``l<i>.norm1`` (``.b``), ``l<i>.ls1``, ``l<i>.mix.*``,
``l<i>.norm2`` (``.b``), ``l<i>.ls2``, ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

from ..config.zepilorn import ZepilornConfig, rotated_dims
from ..parts.base import PartSpec
from ..parts.model import LayerCall, ModelSpec
from ..registry import register_architecture

_NAMES = {"norm1": "norm1", "mixer": "mix.", "norm2": "norm2", "ffn": "mlp.", "scale1": "ls1", "scale2": "ls2"}
SINK_LOGIT = 0.0         # the attention's softmax has one more in its denominator


def _mixer(cfg: ZepilornConfig, layer: dict) -> PartSpec:
    m = layer["mixer"]
    sizes = {"hidden_size": cfg.width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "eps": cfg.norm_eps}
    window = (m.get("mask") or {}).get("size")
    if layer["type"] == "attention":
        dims = rotated_dims(m)
        rot = m.get("rot") or {}
        return PartSpec("head_normed_attention", {
            **sizes, "kv_heads": m["kv_heads"], "scale": m["scale"], "qk_norm": "after", "window": window,
            "position": PartSpec("rope_yarn_neox", {"head_dim": m["dim"], "theta": rot["base"], "rotary_dim": dims,
                                                    "scaling": rot.get("scaling")}) if dims else None,
            "sink_logit": SINK_LOGIT, "own_kv": m.get("kv_from") is None})
    if layer["type"] == "latent_attention":
        return PartSpec("latent_attention", {
            **sizes, "rot_dim": 0, "kv_rank": m["kv_rank"], "q_rank": None, "rope_base": 1.0, "window": window,
            "scale": m["scale"], "sink": False, "gate": False})
    return PartSpec("retention", {**sizes, "decay": m["decay"], "activation": "silu", "key_scale": 1.0, "norm": "all",
                                  "norm_weight": True, "gate": "sigmoid"})


def build_spec(cfg: ZepilornConfig) -> ModelSpec:
    norm = PartSpec("layernorm", {"size": cfg.width, "eps": cfg.norm_eps, "param": ""})
    layers, prefixes, order = [], [], []
    for i, layer in enumerate(cfg.layers):
        mlp = layer.get("mlp")
        ffn = PartSpec("swiglu_dense", {"hidden_size": cfg.width, "intermediate_size": mlp["ff"], "activation": "gelu_tanh",
                                        "names": {"gate": "gate", "up": "up", "down": "down"}}) if mlp is not None else None
        layers.append(PartSpec("postnorm", {"norm1": norm, "mixer": _mixer(cfg, layer),
                                            "norm2": norm if ffn is not None else None, "ffn": ffn,
                                            "hidden_size": cfg.width, "layer_scale": True, "names": _NAMES}))
        prefixes.append(f"l{i}.")
        order.append(LayerCall(i, reads_cache_of=layer["mixer"].get("kv_from") if layer["type"] == "attention" else None))
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, layers=layers, layer_prefixes=prefixes,
                     final_norm=norm, final_norm_prefix="final.norm", embed_name="embed", lm_head_name="head", order=order,
                     # ordinary launches, as Faguzen's steps: a dependent launch around the paired product kernel has
                     # stopped answering there and the cause is not known
                     dependent_launch=False)


register_architecture(ZepilornConfig.architecture, ZepilornConfig, build_spec, model_type=ZepilornConfig.model_type)

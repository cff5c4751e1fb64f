"""Gakenex as a ``ModelSpec`` of parts.

Token embedding (which is also the head) plus a learned vector per position, normed; layers that norm their input once
and add mixer and feed-forward of it side by side; a capped head.  Norms store their weight's distance from one.  The
mixer is attention whose heads are the difference of two score maps over the same values, with a short convolution over
time on queries, keys and values, a norm per map, no positions in the scores, a window that keeps the first tokens, and a
gate per output entry.  Feed-forward: a gated MLP with clamped halves, or experts chosen by sigmoid scores that weigh
what an expert takes in, or none.
Tensor names are the checkpoint's own: ``embed``, ``pos``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm``.
"""
from __future__ import annotations

from ..config.gakenex import GakenexConfig
from ..parts.base import PartSpec
from ..parts.model import ModelSpec
from ..registry import register_architecture

_NAMES = {"norm1": "norm1", "mixer": "mix.", "ffn": "mlp."}
GLU_ALPHA, GLU_SHIFT = 1.702, 1.0        # of the clamped gate


def _mixer(cfg: GakenexConfig, m: dict) -> PartSpec:
    mask = m.get("mask") or {}
    return PartSpec("differential_attention", {
        "hidden_size": cfg.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
        "scale": m["scale"], "eps": cfg.norm_eps, "diff": m["diff"], "conv_taps": m.get("conv"),
        "window": mask.get("size"), "keep_first": mask.get("keep_first") or 0, "gate": True})


def _ffn(cfg: GakenexConfig, mlp: dict | None) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("clamped_glu_dense", {"hidden_size": cfg.width, "intermediate_size": mlp["ff"], "limit": mlp["limit"],
                                              "alpha": GLU_ALPHA, "shift": GLU_SHIFT})
    router = mlp["router"]
    return PartSpec("moe_topk", {
        "hidden_size": cfg.width, "num_experts": router["experts"], "top_k": router["top"],
        "expert_intermediate_size": mlp["expert"]["ff"], "norm_topk_prob": False, "score": "sigmoid", "weigh": "input",
        "names": {"router": "router", "gate": "e{e}.gate", "up": "e{e}.up", "down": "e{e}.down"}})


def build_spec(cfg: GakenexConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "param": "", "offset": 1.0})
    layers, prefixes = [], []
    for i, layer in enumerate(cfg.layers):
        layers.append(PartSpec("parallel", {"norm1": norm, "mixer": _mixer(cfg, layer["mixer"]),
                                            "ffn": _ffn(cfg, layer.get("mlp")), "names": _NAMES}))
        prefixes.append(f"l{i}.")
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, layers=layers, layer_prefixes=prefixes, final_norm=norm,
                     final_norm_prefix="final.norm", embed_name="embed", lm_head_name=None, tie_word_embeddings=True,
                     embed_position=PartSpec("learned", {"max_positions": cfg.max_positions, "hidden_size": cfg.width,
                                                         "param": ""}), embed_position_prefix="pos",
                     embed_norm=norm, embed_norm_prefix="embed.norm", logit_softcap=cfg.logit_softcap,
                     # ordinary launches, as the other designs whose products run paired: a dependent launch around the
                     # paired product kernel has stopped answering in one of them and the cause is not known
                     dependent_launch=False)


register_architecture(GakenexConfig.architecture, GakenexConfig, build_spec, model_type=GakenexConfig.model_type)

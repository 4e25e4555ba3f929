"""Zirivik as data: its configuration turned into a ``ModelSpec``.

Every layer is a sandwich block (a norm before and after each sublayer, all with weights stored
around zero that enter as ``1 + w``).  Its mixer is the lightning part in the variant "no
activations, rotate-half rotation of q and k, keys times ``dim^(-1/2)``, a norm per head without
weight, a SiLU gate" (``retention`` layers), or the attention part without position encoding, with a
window and the sequence's first tokens kept (``attention`` layers; with ``kv_from`` a layer has no
key and value projections and its run reads the cache of the named layer's run).  The feed-forward
is the dense one with the squared ReLU, or the routed part in the variant "sigmoid scores, no
correction, no groups, clamped gated experts, the weight on the expert's input".  The head is the
embedding table (without the embedding's scale); the logits are soft-capped.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.norm1``, ``norm1b``, ``norm2``,
``norm2b``; ``l<i>.mix.{q, k, v, g, o}`` (attention has no ``g``); ``l<i>.mlp.{up, down}`` or
``l<i>.mlp.{router, e<j>.gate, e<j>.up, e<j>.down}``; matrices are ``[out, in]``.
"""
from __future__ import annotations

from typing import Any, Dict

from ..config.zirivik import ZirivikConfig, ZirivikDense
from ..parts.base import LayerSpec, ModelSpec, PartSpec, RunSpec

NORM_OFFSET = 1.0       # the norms' weights are stored around zero
GATE_SLOPE = 1.702      # sigmoid(1.702 g) in an expert's gate
UP_SHIFT = 1.0          # an expert's up branch enters as (u + 1)


def zirivik_spec(cfg: ZirivikConfig) -> ModelSpec:
    norm = PartSpec("rms", {"width": cfg.width, "eps": cfg.eps, "offset": NORM_OFFSET})
    layers, schedule, unused = [], [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        src = None
        names = {"norm1.weight": p + "norm1", "norm1b.weight": p + "norm1b",
                 "mixer.q_proj": p + "mix.q", "mixer.o_proj": p + "mix.o"}
        if layer.type == "retention":
            position = None
            if m.rot_base is not None:
                position = PartSpec("rotary", {"theta": m.rot_base, "rot_dim": m.rot_dims, "pairing": "half"})
            mixer = PartSpec("lightning", {
                "width": cfg.width, "n_heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": m.decay, "eps": cfg.eps,
                "activation": None, "position": position, "k_scale": m.dim ** -0.5, "norm": "head", "gate": "silu"})
            names.update({"mixer.k_proj": p + "mix.k", "mixer.v_proj": p + "mix.v", "mixer.g_proj": p + "mix.g"})
        else:
            src = m.kv_from
            mixer = PartSpec("attention", {
                "width": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim,
                "eps": cfg.eps, "scale": m.scale, "window": m.window, "keep_first": m.keep_first, "own_kv": src is None,
                "exact_weights": True})
            if src is None:
                names.update({"mixer.k_proj": p + "mix.k", "mixer.v_proj": p + "mix.v"})
        params = {"norm1": norm, "mixer": mixer, "norm1b": norm}
        f = layer.mlp
        if f is not None:
            q = p + "mlp."
            names.update({"norm2.weight": p + "norm2", "norm2b.weight": p + "norm2b"})
            if isinstance(f, ZirivikDense):
                ffn = PartSpec("dense_mlp", {"width": cfg.width, "inner": f.ff, "activation": "relu_squared", "bias": False})
                names.update({"ffn.up_proj": q + "up", "ffn.down_proj": q + "down"})
            else:
                ffn = PartSpec("mixture_of_experts", {
                    "width": cfg.width, "n_experts": f.experts, "top": f.top, "inner": f.ff, "correction": False,
                    "score": "sigmoid", "gate_alpha": GATE_SLOPE, "limit": f.limit, "up_shift": UP_SHIFT,
                    "weight_on": "input"})
                names["ffn.router"] = q + "router"
                for e in range(f.experts):
                    for kind in ("gate", "up", "down"):
                        names[f"ffn.experts.{e}.{kind}_proj"] = f"{q}e{e}.{kind}"
            params.update({"norm2": norm, "norm2b": norm, "ffn": ffn})
        else:       # a checkpoint may still carry the norms of the feed-forward the layer does not have
            unused += [p + "norm2", p + "norm2b"]
        layers.append(LayerSpec(block=PartSpec("sandwich", params), names=names))
        schedule.append(RunSpec(layer=i, cache_of=src))         # run i is layer i: every layer runs once, in order
    return ModelSpec(
        vocab_size=cfg.vocab, width=cfg.width, embedding_name="embed", layers=tuple(layers), schedule=tuple(schedule),
        final_norm=norm, final_norm_names={"weight": "final.norm"}, head_name=None, ignored_names=tuple(unused),
        max_positions=cfg.max_positions, stop_ids=tuple(cfg.eos_token_ids), embedding_scale=cfg.embedding_scale,
        logit_softcap=cfg.logit_softcap)


def describe(config: Dict[str, Any]) -> ModelSpec:
    return zirivik_spec(ZirivikConfig.from_dict(config))

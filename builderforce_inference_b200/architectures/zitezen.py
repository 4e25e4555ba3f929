"""Zitezen as data: its configuration turned into a ``ModelSpec``.

Every layer is a hyper block (copies of the residual stream, read and renewed around each sublayer) with
dynamic tanh norms and a scale per channel on each sublayer's output.  Its mixer is the matrix memory
part (``mlstm`` layers); the latent attention part in the variant "query latent, rotation of adjacent
pairs" (``latent_attention``); or the weighted sum of two members side by side (``parallel``): the attention
part in the variant "norm per head before a rotate-half rotation of the first ``rot.dims`` values, value
heads of their own size, soft-capped scores, a gate per head", and the matrix memory.  The feed-forward,
where a layer has one, is the dense part with the squared ReLU.  A loop is a schedule in which the same
layers appear several times, every run with a cache and a state of its own.  The head is a tensor of its
own and sees the norm of the copies' sum.

Tensor names: ``embed``, ``head``, ``final.norm`` (with ``.alpha`` and ``.b``, as every norm), and per layer
``l<i>.norm1``, ``norm2``, ``ls1``, ``ls2``, ``hc1.{in, out, mix}``, ``hc2.{in, out, mix}``; ``l<i>.mix.*`` (matrix
memory: ``q, k, v, g, i, i.b, f, f.b, norm, o``; latent attention: ``dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o``;
parallel: ``left.{q, k, v, q.norm, k.norm, g, o}`` and the memory's under ``right``); ``l<i>.mlp.{up, down}``;
matrices are ``[out, in]``.
"""
from __future__ import annotations

from typing import Any, Dict

from ..config.zitezen import ZitezenConfig, ZitezenLatent, ZitezenMemory
from ..parts.base import LayerSpec, ModelSpec, PartSpec, RunSpec


def _rotary(rot, pairing: str):
    return None if rot is None else PartSpec("rotary", {"theta": rot.base, "rot_dim": rot.dims, "pairing": pairing})


def _memory(cfg: ZitezenConfig, m: ZitezenMemory, local: str, stored: str):
    part = PartSpec("mlstm", {"width": cfg.width, "n_heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap,
                              "eps": cfg.eps})
    names = {f"{local}{n}_proj": stored + n for n in ("q", "k", "v", "g", "i", "f", "o")}
    names.update({f"{local}i_proj.bias": stored + "i.b", f"{local}f_proj.bias": stored + "f.b", f"{local}norm": stored + "norm"})
    return part, names


def _norm_names(local: str, stored: str) -> Dict[str, str]:
    prefix = local + "." if local else ""
    return {prefix + "weight": stored, prefix + "bias": stored + ".b", prefix + "alpha": stored + ".alpha"}


def zitezen_spec(cfg: ZitezenConfig) -> ModelSpec:
    norm = PartSpec("dynamic_tanh", {"width": cfg.width})
    layers, unused = [], []
    for i, layer in enumerate(cfg.layers):
        p, q, m = f"l{i}.", f"l{i}.mix.", layer.mixer
        names = _norm_names("norm1", p + "norm1")
        if isinstance(m, ZitezenMemory):
            mixer, more = _memory(cfg, m, "mixer.", q)
        elif isinstance(m, ZitezenLatent):
            mixer = PartSpec("latent_attention", {
                "width": cfg.width, "n_heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "v_dim": m.vdim, "kv_rank": m.kv_rank,
                "q_rank": m.q_rank, "position": _rotary(m.rot, "adjacent"), "eps": cfg.eps, "scale": m.scale})
            more = {"mixer.dq_proj": q + "dq", "mixer.dq_norm": q + "dq.norm", "mixer.uq_proj": q + "uq", "mixer.dkv_proj": q + "dkv",
                    "mixer.dkv_norm": q + "dkv.norm", "mixer.uk_proj": q + "uk", "mixer.uv_proj": q + "uv", "mixer.o_proj": q + "o"}
        else:
            a = m.left
            left = PartSpec("attention", {
                "width": cfg.width, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_dim": a.vdim,
                "position": _rotary(a.rot, "half"), "qk_norm": "head", "eps": cfg.eps, "scale": a.scale, "softcap": a.softcap,
                "gate": "head", "exact_weights": True})
            right, more = _memory(cfg, m.right, "mixer.right.", q + "right.")
            mixer = PartSpec("weighted_sum", {"members": {"left": left, "right": right},
                                              "scales": {"left": m.left_scale, "right": m.right_scale}})
            more.update({f"mixer.left.{n}_proj": f"{q}left.{n}" for n in ("q", "k", "v", "g", "o")})
            more.update({"mixer.left.q_norm": q + "left.q.norm", "mixer.left.k_norm": q + "left.k.norm"})
        names.update(more)
        params = {"width": cfg.width, "streams": cfg.streams, "norm1": norm, "mixer": mixer, "layer_scale": True}
        if layer.ff is not None:
            params.update({"norm2": norm, "ffn": PartSpec("dense_mlp", {"width": cfg.width, "inner": layer.ff,
                                                                        "activation": "relu_squared", "bias": False})})
            names.update(_norm_names("norm2", p + "norm2"))
            names.update({"ffn.up_proj": p + "mlp.up", "ffn.down_proj": p + "mlp.down"})
        for s in ("1", "2"):
            stored = {"read" + s: f"{p}hc{s}.in", "write" + s: f"{p}hc{s}.out", "mix" + s: f"{p}hc{s}.mix", "scale" + s: f"{p}ls{s}"}
            if s == "1" or layer.ff is not None:
                names.update(stored)
            else:       # a checkpoint may still carry what stands around the feed-forward the layer does not have
                unused += list(stored.values()) + list(_norm_names("", p + "norm2").values())
        layers.append(LayerSpec(block=PartSpec("hyper", params), names=names))
    return ModelSpec(
        vocab_size=cfg.vocab, width=cfg.width, embedding_name="embed", layers=tuple(layers),
        schedule=tuple(RunSpec(layer=i) for i in cfg.order), final_norm=norm, final_norm_names=_norm_names("", "final.norm"),
        head_name="head", ignored_names=tuple(unused), max_positions=cfg.max_positions, stop_ids=tuple(cfg.eos_token_ids),
        streams=cfg.streams)


def describe(config: Dict[str, Any]) -> ModelSpec:
    return zitezen_spec(ZitezenConfig.from_dict(config))

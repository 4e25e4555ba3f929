"""``ZirivikConfig``: the sizes and constants of a Zirivik decoder, read from its config.json.

A Zirivik model is a stack of blocks with a norm before and after each sublayer, whose mixer is,
layer by layer, retention (linear attention with a fixed decay per head, rotary positions and a norm
per head) or softmax attention without positions over a sliding window and the sequence's first
tokens; an attention layer may read another one's keys and values.  The feed-forward, where a layer
has one, is dense (squared ReLU) or a mixture of experts whose weights scale the experts' inputs.
config.json carries:

    architecture        "Zirivik"
    vocab, width        vocabulary size, residual width
    norm.eps            epsilon of every RMS norm
    embedding.scale     factor on the embedded tokens (default 1)
    logit_softcap       c in c * tanh(logits / c); absent: the logits as they are
    layers[i].type      "retention" | "attention"
    layers[i].mixer     retention: heads, dim, vdim, decay (one number per head), rot.{base, dims}
                        attention: heads, kv_heads, dim, vdim, scale, mask.{size, keep_first},
                                   kv_from (optional: the earlier attention layer whose keys and values it reads)
    layers[i].mlp       null, or {kind: "dense", ff}, or {kind: "moe", expert.{ff, limit}, router.{experts, top}}

Every value is checked here, so a bad folder fails by key before any weight is read.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, ConfigReader
from .datasun import _sub


@dataclass(frozen=True)
class ZirivikRetention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_base: Optional[float]
    rot_dims: int


@dataclass(frozen=True)
class ZirivikAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    keep_first: int
    kv_from: Optional[int]


@dataclass(frozen=True)
class ZirivikDense:
    ff: int


@dataclass(frozen=True)
class ZirivikMoE:
    experts: int
    top: int
    ff: int
    limit: Optional[float]


@dataclass(frozen=True)
class ZirivikLayer:
    type: str
    mixer: Any
    mlp: Any


def _retention(r: ConfigReader) -> ZirivikRetention:
    heads = r.integer("heads", minimum=1)
    dim = r.integer("dim", minimum=1)
    vdim = r.integer("vdim", default=dim, minimum=1)
    decay = r.raw("decay")
    if not isinstance(decay, (list, tuple)) or len(decay) != heads or \
            not all(isinstance(x, (int, float)) and not isinstance(x, bool) and 0.0 <= x <= 1.0 for x in decay):
        raise ConfigError(f"{r.what}: key 'decay' must list one number from 0 to 1 per head ({heads})")
    base, dims = None, 0
    rot = _sub(r, "rot", required=False)
    if rot is not None:
        dims = rot.integer("dims", minimum=2)
        if dims % 2 != 0 or dims > dim:
            raise ConfigError(f"{rot.what}: key 'dims' must be even and at most dim {dim}, got {dims}")
        base = rot.number("base", positive=True)
    return ZirivikRetention(heads=heads, dim=dim, vdim=vdim, decay=tuple(float(x) for x in decay), rot_base=base, rot_dims=dims)


def _attention(r: ConfigReader, earlier: List[ZirivikLayer]) -> ZirivikAttention:
    heads = r.integer("heads", minimum=1)
    kv = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv != 0:
        raise ConfigError(f"{r.what}: {heads} query heads do not divide into kv_heads {kv}")
    dim = r.integer("dim", minimum=2)
    if dim % 2 != 0 or dim > 512:
        raise ConfigError(f"{r.what}: key 'dim' must be even and at most 512, got {dim}")
    vdim = r.integer("vdim", default=dim, minimum=1)
    if vdim > 512:
        raise ConfigError(f"{r.what}: key 'vdim' must be at most 512, got {vdim}")
    window, keep = None, 0
    mask = _sub(r, "mask", required=False)
    if mask is not None:
        window = mask.integer("size", minimum=1)
        keep = mask.integer("keep_first", default=0, minimum=0)
    src = r.integer("kv_from", default=None, minimum=0)
    if src is not None:
        if src >= len(earlier) or not isinstance(earlier[src].mixer, ZirivikAttention):
            raise ConfigError(f"{r.what}: key 'kv_from' must name an earlier attention layer, got {src}")
        m = earlier[src].mixer
        if m.kv_from is not None:
            raise ConfigError(f"{r.what}: key 'kv_from' names layer {src}, which has no keys and values of its own")
        if (m.heads, m.kv_heads, m.dim, m.vdim) != (heads, kv, dim, vdim):
            raise ConfigError(f"{r.what}: key 'kv_from': layer {src} has other heads, kv_heads, dim or vdim")
    return ZirivikAttention(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=r.number("scale", default=dim ** -0.5),
                            window=window, keep_first=keep, kv_from=src)


def _mlp(r: ConfigReader) -> Any:
    kind = r.string("kind")
    if kind == "dense":
        return ZirivikDense(ff=r.integer("ff", minimum=1))
    if kind != "moe":
        raise ConfigError(f"{r.what}: key 'kind' must be \"dense\" or \"moe\", got {kind!r}")
    router, expert = _sub(r, "router"), _sub(r, "expert")
    experts = router.integer("experts", minimum=1)
    top = router.integer("top", minimum=1)
    if top > experts:
        raise ConfigError(f"{router.what}: key 'top' {top} exceeds the {experts} experts")
    return ZirivikMoE(experts=experts, top=top, ff=expert.integer("ff", minimum=1),
                      limit=expert.number("limit", default=None, positive=True))


@dataclass(frozen=True)
class ZirivikConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: Optional[float]
    layers: Tuple[ZirivikLayer, ...]
    max_positions: int
    eos_token_ids: Tuple[int, ...]

    @classmethod
    def from_dict(cls, data: Dict[str, Any], what: str = "config.json") -> "ZirivikConfig":
        r = ConfigReader(data, what)
        vocab = r.integer("vocab", minimum=1)
        width = r.integer("width", minimum=1)
        eps = _sub(r, "norm").number("eps", positive=True)
        emb = _sub(r, "embedding", required=False)
        scale = emb.number("scale", default=1.0) if emb is not None else 1.0
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(f"{what}: key 'layers' must be a non-empty list")
        layers: List[ZirivikLayer] = []
        for i, entry in enumerate(raw_layers):
            lr = ConfigReader(entry, f"{what}: layers[{i}]")
            kind = lr.string("type")
            mixer = _sub(lr, "mixer")
            if kind == "retention":
                m = _retention(mixer)
            elif kind == "attention":
                m = _attention(mixer, layers)
            else:
                raise ConfigError(f"{lr.what}: key 'type' must be \"retention\" or \"attention\", got {kind!r}")
            mr = _sub(lr, "mlp", required=False)
            layers.append(ZirivikLayer(type=kind, mixer=m, mlp=None if mr is None else _mlp(mr)))
        return cls(vocab=vocab, width=width, eps=eps, embedding_scale=scale,
                   logit_softcap=r.number("logit_softcap", default=None, positive=True), layers=tuple(layers),
                   max_positions=r.integer("max_positions", default=0, minimum=0),
                   eos_token_ids=tuple(r.int_or_list("eos_token_id")))

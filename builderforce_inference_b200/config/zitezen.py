"""``ZitezenConfig``: the sizes and constants of a Zitezen decoder, read from its config.json.

A Zitezen model holds its residual stream several times; every sublayer reads a weighted sum of the
copies through a norm without statistics (dynamic tanh), and its output, scaled per channel, is written
back while the copies are mixed among themselves.  The mixer of a layer is a matrix memory (mLSTM),
latent attention whose queries go through a latent too, or soft-capped grouped-query attention and a
matrix memory side by side; the feed-forward, where a layer has one, is a dense one with the squared
ReLU.  A range of layers may run several times in a row, each time with state of its own.  config.json
carries:

    architecture            "Zitezen"
    vocab, width, streams   vocabulary size, residual width, copies of the residual stream
    norm.eps                epsilon of the RMS norms inside the mixers
    loop                    null or {start, stop, times}: layers start .. stop-1 run `times` times in a row
    layers[i].type          "mlstm" | "latent_attention" | "parallel"
    layers[i].mixer         mlstm: heads, dim, vdim, gate_cap
                            latent_attention: heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot.{base, dims}
                            parallel: left.{heads, kv_heads, dim, vdim, scale, softcap, rot.{base, dims}}, left_scale,
                                      right.{heads, dim, vdim, gate_cap}, right_scale
    layers[i].mlp           null or {kind: "dense", ff}

Every value is checked here, so a bad folder fails by key before any weight is read.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ConfigReader
from .datasun import _sub

MAX_STREAMS = 32        # the kernels keep a channel's copies in registers


@dataclass(frozen=True)
class ZitezenRotation:
    base: float
    dims: int


@dataclass(frozen=True)
class ZitezenMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ZitezenLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Optional[ZitezenRotation]


@dataclass(frozen=True)
class ZitezenAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    rot: Optional[ZitezenRotation]


@dataclass(frozen=True)
class ZitezenParallel:
    left: ZitezenAttention
    right: ZitezenMemory
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class ZitezenLayer:
    type: str
    mixer: Any                  # ZitezenMemory, ZitezenLatent or ZitezenParallel
    ff: Optional[int]           # None: no feed-forward


def _rotation(r: ConfigReader, limit: int) -> Optional[ZitezenRotation]:
    rot = _sub(r, "rot", required=False)
    if rot is None or limit < 2:
        return None
    dims = rot.integer("dims", default=limit, minimum=2)
    if dims % 2 != 0 or dims > limit:
        raise ConfigError(f"{rot.what}: key 'dims' must be even and at most {limit}, got {dims}")
    return ZitezenRotation(base=rot.number("base", positive=True), dims=dims)


def _memory(r: ConfigReader) -> ZitezenMemory:
    dim = r.integer("dim", minimum=1)
    return ZitezenMemory(heads=r.integer("heads", minimum=1), dim=dim, vdim=r.integer("vdim", default=dim, minimum=1),
                         gate_cap=r.number("gate_cap", positive=True))


def _latent(r: ConfigReader) -> ZitezenLatent:
    dim = r.integer("dim", minimum=1)
    rot_dim = r.integer("rot_dim", default=0, minimum=0)
    rank = r.integer("kv_rank", minimum=1)
    if (rank + rot_dim) % 2 != 0 or rank + rot_dim > 1024 or rank > 512:
        raise ConfigError(f"{r.what}: kv_rank = {rank} must be at most 512, kv_rank + rot_dim = {rank + rot_dim} even and at most 1024")
    return ZitezenLatent(heads=r.integer("heads", minimum=1), dim=dim, rot_dim=rot_dim, vdim=r.integer("vdim", default=dim, minimum=1),
                         kv_rank=rank, q_rank=r.integer("q_rank", minimum=1),
                         scale=r.number("scale", default=(dim + rot_dim) ** -0.5, positive=True), rot=_rotation(r, rot_dim))


def _attention(r: ConfigReader) -> ZitezenAttention:
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
    return ZitezenAttention(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=r.number("scale", default=dim ** -0.5, positive=True),
                            softcap=r.number("softcap", default=None, positive=True), rot=_rotation(r, dim))


def _layer(r: ConfigReader) -> ZitezenLayer:
    kind, m = r.string("type"), _sub(r, "mixer")
    if kind == "mlstm":
        mixer: Any = _memory(m)
    elif kind == "latent_attention":
        mixer = _latent(m)
    elif kind == "parallel":
        mixer = ZitezenParallel(left=_attention(_sub(m, "left")), right=_memory(_sub(m, "right")),
                                left_scale=m.number("left_scale", default=1.0), right_scale=m.number("right_scale", default=1.0))
    else:
        raise ConfigError(f"{r.what}: key 'type' must be \"mlstm\", \"latent_attention\" or \"parallel\", got {kind!r}")
    f = _sub(r, "mlp", required=False)
    ff = None
    if f is not None:
        ff_kind = f.string("kind", default="dense")
        if ff_kind != "dense":
            raise ConfigError(f"{f.what}: key 'kind' must be \"dense\", got {ff_kind!r}")
        ff = f.integer("ff", minimum=1)
    return ZitezenLayer(type=kind, mixer=mixer, ff=ff)


@dataclass(frozen=True)
class ZitezenConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    layers: Tuple[ZitezenLayer, ...]
    loop: Optional[Tuple[int, int, int]]        # start, stop, times
    max_positions: int
    eos_token_ids: Tuple[int, ...]

    @property
    def order(self) -> Tuple[int, ...]:
        """The layers in the order they run."""
        n = len(self.layers)
        start, stop, times = self.loop if self.loop is not None else (0, 0, 0)
        return tuple(range(start)) + tuple(range(start, stop)) * times + tuple(range(stop, n))

    @classmethod
    def from_dict(cls, data: Dict[str, Any], what: str = "config.json") -> "ZitezenConfig":
        r = ConfigReader(data, what)
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        streams = r.integer("streams", default=1, minimum=1)
        if streams > MAX_STREAMS:
            raise ConfigError(f"{what}: key 'streams' must be at most {MAX_STREAMS}, got {streams}")
        raw = r.raw("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError(f"{what}: key 'layers' must be a non-empty list")
        layers = tuple(_layer(ConfigReader(entry, f"{what}: layers[{i}]")) for i, entry in enumerate(raw))
        loop = None
        lr = _sub(r, "loop", required=False)
        if lr is not None:
            start, stop = lr.integer("start", minimum=0), lr.integer("stop", minimum=0)
            if not start <= stop <= len(layers):
                raise ConfigError(f"{lr.what}: layers {start} to {stop} are no range of the {len(layers)} layers")
            loop = (start, stop, lr.integer("times", minimum=1))
        return cls(vocab=vocab, width=width, streams=streams, eps=_sub(r, "norm").number("eps", positive=True), layers=layers,
                   loop=loop, max_positions=r.integer("max_positions", default=0, minimum=0),
                   eos_token_ids=tuple(r.int_or_list("eos_token_id")))

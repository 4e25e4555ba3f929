"""Linear attention with a decay per head ("lightning attention"), as a mixer.

With ``q = silu(W_q h)``, ``k = silu(W_k h)`` (``heads x dim``) and ``v = silu(W_v h)``
(``heads x vdim``), every head keeps a ``dim x vdim`` state per sequence:

    S_t = decay_h * S_(t-1) + k_t v_t^T        o_t = S_t^T q_t

The heads of a token are RMS-normed together (one weight over ``heads * vdim``), multiplied by
``sigmoid(W_g h)`` and projected by ``W_o`` into the residual stream.  The state is float32, zero
when a slot is taken (the cache clears it), and the only thing a sequence keeps: a step may bring
whole prompts, further pieces of one, or single tokens.

The four input projections are one matrix product over the concatenated weights; the activations
are applied where the values are read (the recurrence kernels, the gated norm), in float32.

Variants, each a parameter: ``activation`` None (q, k and v as projected); ``position`` (a rotate-half
encoding of the first values of every q and k head by the token's position, after the activation) and
``k_scale`` (a factor on k, after the rotation), both applied in float32 by the kernels that read q and
k; ``norm`` ``"head"`` (every head's output divided by its own root mean square, without a weight);
``gate`` ``"silu"`` (``silu(W_g h)``).  Retention is the combination of the four.
"""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch

from ..kernels import ops
from ..kernels.linear import EPI_ACCUMULATE, EPI_STORE, linear
from .base import MIXERS, POSITION_ENCODINGS, Mixer, ParamSpec, PartSpec, StateNeed


@MIXERS.register("lightning")
class LightningAttention(Mixer):
    graph_safe = True

    def __init__(self, width: int, n_heads: int, dim: int, vdim: int, decay: Sequence[float], eps: float = 1e-6,
                 activation: Optional[str] = "silu", position: Optional[PartSpec] = None, k_scale: float = 1.0,
                 norm: str = "row", gate: str = "sigmoid"):
        if n_heads < 1 or dim < 1 or vdim < 1:
            raise ValueError(f"lightning attention: bad sizes heads={n_heads} dim={dim} vdim={vdim}")
        if len(decay) != n_heads:
            raise ValueError(f"lightning attention: {len(decay)} decays for {n_heads} heads")
        self.width, self.n_heads, self.dim, self.vdim = int(width), int(n_heads), int(dim), int(vdim)
        if activation not in ("silu", None) or norm not in ("row", "head") or gate not in ("sigmoid", "silu"):
            raise ValueError(f"lightning attention: activation {activation!r}, norm {norm!r}, gate {gate!r}")
        if norm == "row" and gate != "sigmoid":
            raise ValueError("lightning attention: the norm over all heads goes with a sigmoid gate")
        self.act = ops.LIGHT_ACT_SILU if activation == "silu" else ops.LIGHT_ACT_NONE
        self.k_scale, self.norm_heads = float(k_scale), norm == "head"
        self.gate_act = ops.GATE_SILU if gate == "silu" else ops.GATE_SIGMOID
        self.position = POSITION_ENCODINGS.build(position if position is not None else PartSpec("none"))
        if getattr(self.position, "pairing", "half") != "half" or getattr(self.position, "rot_dim", 0) > dim:
            raise ValueError("lightning attention: q and k turn by halves of at most a head's values")
        self.decay_values = tuple(float(x) for x in decay)
        self.eps = float(eps)
        self.w_in = self.w_o = self.norm = self.decay = None

    def children(self):
        return {"position": self.position}

    def prepare(self, runtime, max_positions: int) -> None:
        self.position.prepare(runtime, max_positions)

    def param_specs(self) -> Dict[str, ParamSpec]:
        qk, vv, w = self.n_heads * self.dim, self.n_heads * self.vdim, self.width
        specs = {"q_proj": ParamSpec((qk, w)), "k_proj": ParamSpec((qk, w)), "v_proj": ParamSpec((vv, w)),
                 "g_proj": ParamSpec((vv, w)), "o_proj": ParamSpec((w, vv))}
        if not self.norm_heads:
            specs["norm"] = ParamSpec((vv,), "norm")
        return specs

    def cache_need(self):
        return StateNeed((self.n_heads, self.dim, self.vdim), "float32")

    def load(self, tensors, runtime) -> None:
        mats = [tensors[n] for n in ("q_proj", "k_proj", "v_proj", "g_proj")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        self.w_in = torch.cat(mats, dim=0).contiguous()
        self.w_o = tensors["o_proj"]
        self.norm = tensors.get("norm")
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=runtime.device)

    def forward(self, ctx, h, residual, run) -> None:
        self._run(ctx, h, residual, run, EPI_ACCUMULATE)

    def forward_store(self, ctx, h, out, run) -> None:
        self._run(ctx, h, out, run, EPI_STORE)

    def _run(self, ctx, h, target, run, epilogue) -> None:
        state = run.state
        if state is None or not run.writes_cache:
            raise RuntimeError("lightning attention needs a state of its own for its run")
        qk, vv = self.n_heads * self.dim, self.n_heads * self.vdim
        proj = ctx.rows("light.proj", 2 * qk + 2 * vv)
        linear(h, self.w_in, proj, EPI_STORE)
        o = ctx.rows("light.o", vv, torch.float32)
        self.recur(ctx, proj, o, state)
        y = ctx.rows("light.y", vv)
        gate = proj[:, 2 * qk + vv:]
        if self.norm_heads:
            ops.gated_group_norm(o, gate, None, self.eps, y, self.n_heads, gate_first=False, gate_act=self.gate_act)
        else:
            ops.gated_rmsnorm(o, gate, self.norm, self.eps, y)
        linear(y, self.w_o, target, epilogue)

    def recur(self, ctx, proj, o, state) -> None:
        qk = self.n_heads * self.dim
        fused = self.position.fused_rotary()
        if fused is None:
            raise RuntimeError("lightning attention needs a position encoding its kernels apply themselves")
        turn = {"act": self.act, "rope_table": fused[0], "rot_dim": fused[1], "token_pos": ctx.token_pos, "k_scale": self.k_scale,
                "status": ctx.status}
        if proj.dtype == torch.bfloat16:
            from ..kernels import fast_ops
            if ctx.max_seq_tokens >= fast_ops.LIGHTNING_CHUNK_MIN_TOKENS and fast_ops.lightning_chunks_bf16(
                    proj, 0, qk, 2 * qk, o, state, self.decay, ctx.cu_seqlens, ctx.seq_slot, ctx.n_seqs,
                    self.n_heads, self.dim, self.vdim, **turn):
                return
        ops.lightning_scan(proj, 0, qk, 2 * qk, o, state, self.decay, ctx.cu_seqlens, ctx.seq_slot, ctx.n_seqs,
                           self.n_heads, self.dim, self.vdim, few_tokens=ctx.max_seq_tokens == 1,
                           single_tokens=ctx.max_seq_tokens == 1 and ctx.n_tokens == ctx.n_seqs, **turn)

"""Zirivik through the package against the plain implementation (tests/plain/zirivik_plain.py): every
mechanism's kernel alone, then whole models with sizes of their own, stepped whole, token by token,
in portions, in unequal batches, over reused slots and pages, and generated from greedily.

Some tests shape their inputs so that one key, one edge or one expert decides the result."""
import json
import math
import os

import pytest
import torch

from attention_pages import Pages
from helpers import rel_err
from plain import zirivik_plain as P
from zirivik_models import BF16, F32, make_weights, model, prompts, random_config, write_folder

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")


def close(got, ref, dtype):
    """Whether a model's output is the plain implementation's.  float32: every value, to 3e-5 of the
    largest.  bfloat16: 95 % of the rows (all but one, of few) lie within 6e-2 and every row is finite and
    within 1, since rounding is amplified where a token is badly conditioned; a lost state, a wrong key or
    a wrong expert shows as 0.3 and more.  The float32 run is the sharp test."""
    if dtype in (F32, "float32"):
        return rel_err(got, ref) < 3e-5
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    if got.shape != ref.shape or not torch.isfinite(got).all():
        return False
    rows = (got - ref).abs().reshape(got.shape[0], -1).max(dim=1).values / max(1e-6, float(ref.abs().max()))
    return int((rows > 6e-2).sum()) <= max(1, rows.numel() // 20) and float(rows.max()) < 1.0


def ops():
    from builderforce_inference_b200.kernels import ops as o
    return o


def i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device=DEV)


def q64(t, dt):
    """The values a tensor of storage type ``dt`` holds, as float64."""
    return t.to(dt).to(torch.float64)


def engine(name, dtype, **kw):
    from builderforce_inference_b200.engine.engine import Engine
    folder, cfg, w = model(name, dtype)
    return Engine.load(folder, dtype=dtype, max_tokens=kw.pop("max_tokens", 2048), **kw), cfg, w


def S(slot, tokens, want=None):
    from builderforce_inference_b200.engine.engine import SequenceStep
    return SequenceStep(slot, tokens, list(range(len(tokens))) if want is None else want)


# ------------------------------------------------------------------------------------------------
# attention: a window and the first positions, in every kernel
# ------------------------------------------------------------------------------------------------
def reference(q, k, v, scale, window, keep, dt):
    n, n_q, _ = q.shape
    return P.masked_attention(q64(q, dt), q64(k, dt), q64(v, dt), scale, P.window_mask(n, window, keep)).reshape(n, -1)


def attend(kind, q, pages, seqs, n_q, dv, scale, dt):
    """One step through the kernel ``kind``: "general", "decode", "short" (mma.sync prompt kernel), "long"
    (tcgen05), or "chosen", the one the attention part takes."""
    from builderforce_inference_b200.engine.context import Workspace, build_context
    from builderforce_inference_b200.kernels import attention as choose
    from builderforce_inference_b200.kernels import fast_ops
    pages.forget({s: st for s, st, _ in seqs})
    ctx = build_context([(s, st, [0] * t) for s, st, t in seqs], dt, Workspace(DEV), DEV)
    qd = q.to(dt).to(DEV).contiguous()
    out = torch.full((qd.shape[0], n_q * dv), float("nan"), dtype=dt, device=DEV)
    if kind == "general":
        ops().attention_paged(qd, qd.stride(0), out, pages.view, ctx.cu_seqlens, ctx.seq_slot, ctx.seq_start, ctx.n_seqs,
                              ctx.max_seq_tokens, n_q, scale)
    elif kind == "decode":
        assert fast_ops.attention_decode_bf16(ctx, qd, out, pages.view, n_q, scale, exact_weights=True)
    elif kind == "short":
        assert fast_ops.attention_prefill_bf16(ctx, qd, out, pages.view, n_q, scale, None, True)
    elif kind == "long":
        assert fast_ops.attention_prefill_tcgen05_bf16(ctx, qd, out, pages.view, n_q, scale, None, True)
    else:
        assert choose.attend(ctx, qd, out, pages.view, n_q, scale, None, True)
    if kind in ("decode", "long", "chosen"):
        assert int(fast_ops.tc_status(DEV)[0]) == 0
    return out.double().cpu()


MASKS = [(9, 3), (70, 130), (64, 64), (1, 5), (65, 1), (128, 127), (40, 0), (300, 200), (1000, 7), (None, 0), (129, 129)]


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n_q,n_kv,d,dv", [(4, 2, 24, 10), (6, 1, 16, 40), (3, 3, 48, 48)])
@pytest.mark.parametrize("window,keep", MASKS)
def test_general_attention_in_a_mixed_batch(dt, n_q, n_kv, d, dv, window, keep):
    g = torch.Generator().manual_seed(n_q * 100 + d)
    seqs = [(2, 0, 150), (0, 330, 1), (1, 261, 7), (3, 0, 2)]       # a prompt, a single token far in, a continuation, two first tokens
    pages = Pages(4, 384, n_kv, d, dv, dt, window, keep)
    qs, refs = [], []
    for slot, start, t in seqs:
        n = start + t
        k, v, q = (torch.randn(n, h, e, generator=g) for h, e in ((n_kv, d), (n_kv, dv), (n_q, d)))
        pages.write(slot, k, v)
        refs.append(reference(q, k, v, 0.2, window, keep, dt)[start:])
        qs.append(q[start:].reshape(t, n_q * d))
    got = attend("general", torch.cat(qs), pages, seqs, n_q, dv, 0.2, dt)
    assert rel_err(got, torch.cat(refs)) < (3e-6 if dt == F32 else 1e-2)


@pytest.mark.parametrize("n_q,n_kv,d", [(8, 2, 64), (4, 1, 128), (40, 2, 64), (2, 2, 128)])
@pytest.mark.parametrize("window,keep", MASKS)
def test_tensor_core_attention_reads_the_window_and_the_first_positions(n_q, n_kv, d, window, keep):
    """The three bfloat16 kernels in unequal batches.  The weights are float32 in effect, so what is left
    is the rounding of the output."""
    g = torch.Generator().manual_seed(n_q + d)
    lens = [700, 131, 1, 449]
    pages = Pages(4, 704, n_kv, d, d, BF16, window, keep)
    data = []
    for slot, n in enumerate(lens):
        k, v, q = (torch.randn(n, h, d, generator=g) for h in (n_kv, n_kv, n_q))
        pages.write(slot, k, v)
        data.append((q, reference(q, k, v, 0.15, window, keep, BF16)))

    def check(kind, seqs):
        got = attend(kind, torch.cat([data[s][0][st:st + t] for s, st, t in seqs]).reshape(-1, n_q * d), pages, seqs, n_q, d, 0.15, BF16)
        ref = torch.cat([data[s][1][st:st + t] for s, st, t in seqs])
        assert float((got - ref.to(BF16).double()).abs().max()) <= 2.0 * float(ref.abs().max()) * 2.0 ** -9, (kind, seqs)

    for kind in ("long", "short", "chosen"):
        check(kind, [(1, 0, 131), (0, 0, 700), (2, 0, 1), (3, 0, 449)])
        check(kind, [(0, 500, 200), (1, 129, 2), (3, 65, 384)])
    for kind in ("decode", "chosen"):
        check(kind, [(0, 699, 1), (1, 130, 1), (2, 0, 1), (3, 448, 1)])
        check(kind, [(3, 64, 1), (1, 63, 1), (0, 9, 1)])


@pytest.mark.parametrize("kind,dt,d", [("general", F32, 16), ("general", BF16, 16), ("decode", BF16, 64), ("short", BF16, 64), ("long", BF16, 64),
                                       ("decode", BF16, 128), ("short", BF16, 128), ("long", BF16, 128)])
@pytest.mark.parametrize("window,keep", [(41, 7), (64, 64), (100, 65), (1, 1), (130, 0)])
def test_one_loud_key_just_inside_and_just_outside_the_window_and_the_first_positions(kind, dt, d, window, keep):
    """Among hundreds of quiet keys one is loud (a large score with every query) and carries a value of its
    own: a query hears it exactly when it lies in the window or among the first positions, in a prompt, in
    a portion of one and as a single decoded token."""
    n_q, n_kv, n = 2, 1, 400
    g = torch.Generator().manual_seed(window)
    for loud in sorted({0, max(0, keep - 1), keep, 200, 255, 256}):
        k, v, q = (0.05 * torch.randn(n, h, d, generator=g) for h in (n_kv, n_kv, n_q))
        k[loud, 0, 0], q[:, :, 0], v[loud, 0, :] = 40.0, 40.0, 7.0
        pages = Pages(1, n, n_kv, d, d, dt, window, keep, seed=loud)
        pages.write(0, k, v)
        ref = reference(q, k, v, 0.25, window, keep, dt)
        spots = sorted({loud, loud + 1, loud + window - 1, loud + window, loud + window + 1, 64, 319, 320, n - 1})
        if kind == "decode":
            runs = [(p, 1) for p in spots if loud <= p < n]
        else:
            runs = [(0, n)] + [(p, min(n - p, c)) for p in spots for c in (2, 130) if loud <= p < n - 1]
        for start, t in runs:
            got = attend(kind, q[start:start + t].reshape(t, -1), pages, [(0, start, t)], n_q, d, 0.25, dt)
            assert rel_err(got, ref[start:start + t]) < (1e-5 if dt == F32 else 1e-2), (loud, start, t)
            for i in range(t):
                heard = abs(float(got[i, 0])) > 3.0
                assert heard == (start + i >= loud and (start + i - loud < window or loud < keep)), (loud, start, i)


# ------------------------------------------------------------------------------------------------
# retention
# ------------------------------------------------------------------------------------------------
def run_retention(kind, proj, H, D, V, seqs, state, decay, table, rot, k_scale, dt, act=0):
    o = ops()
    cu, pos = [0], []
    for _, st, t in seqs:
        cu.append(cu[-1] + t)
        pos += range(st, st + t)
    out = torch.full((cu[-1], H * V), float("nan"), dtype=F32, device=DEV)
    args = (proj.to(dt).to(DEV), 0, H * D, 2 * H * D, out, state, decay.float().to(DEV), i32(cu), i32([s for s, _, _ in seqs]), len(seqs), H, D, V)
    kw = dict(act=act, rope_table=table, rot_dim=rot, token_pos=i32(pos), k_scale=k_scale, status=torch.zeros(1, dtype=torch.int32, device=DEV))
    if kind == "chunks":
        from builderforce_inference_b200.kernels import fast_ops
        assert fast_ops.lightning_chunks_bf16(*args, **kw)
    else:
        single = all(t == 1 for _, _, t in seqs)
        o.lightning_scan(*args, few_tokens=single, single_tokens=single, **kw)
    assert int(kw["status"]) == 0
    return out.double().cpu()


def plain_retention(proj, H, D, V, decay, start, rot, base, k_scale, dt, state=None):
    x, n = q64(proj, dt), proj.shape[0]
    q, k = x[:, :H * D].reshape(n, H, D), x[:, H * D:2 * H * D].reshape(n, H, D)
    if rot:
        q, k = (P.rotate_half(y, range(start, start + n), base, rot) for y in (q, k))
    o, S_end = P.decayed_recurrence(q, k * k_scale, x[:, 2 * H * D:].reshape(n, H, V), decay.float().double(), state)
    return o.reshape(n, H * V), S_end


@pytest.mark.parametrize("kind,dt,sizes", [("scan", F32, (3, 10, 6, 6)), ("scan", BF16, (2, 24, 40, 24)), ("scan", F32, (1, 260, 33, 64)),
                                           ("scan", BF16, (2, 64, 1, 0)), ("chunks", BF16, (2, 64, 64, 64)), ("chunks", BF16, (3, 128, 32, 48)),
                                           ("chunks", BF16, (1, 48, 16, 16)), ("chunks", BF16, (2, 16, 128, 0)), ("chunks", BF16, (40, 128, 128, 128))])
def test_retention_whole_in_portions_and_token_by_token(kind, dt, sizes):
    """Rotation, key scale and recurrence are float32 (in effect) in every kernel: only rounded inputs enter."""
    from builderforce_inference_b200.parts.rotary import rotary_table
    H, D, V, rot = sizes
    n, base, ks = (203, 300.0, D ** -0.5) if H < 40 else (70, 1e4, D ** -0.5)
    g = torch.Generator().manual_seed(H * D + V)
    proj = torch.randn(n, 2 * H * D + H * V, generator=g)
    decay = torch.tensor([(0.0, 0.5, 0.97, 0.9995)[h % 4] if H > 1 else 0.99 for h in range(H)])
    table = rotary_table(base, rot, 256, DEV) if rot else None
    ref, S_ref = plain_retention(proj, H, D, V, decay, 0, rot, base, ks, dt)
    cut_lists = [[n], [64, 1, 2, n - 67]] + ([[1] * n] if H < 40 else [])
    for cuts in cut_lists:
        state = torch.zeros(3, H, D, V, dtype=F32, device=DEV)
        state[0].fill_(float("nan"))                     # another slot's state must not matter
        outs, at = [], 0
        for c in cuts:
            how = kind if c > 1 else "scan"              # single tokens have a kernel of their own, behind the same face
            outs.append(run_retention(how, proj[at:at + c], H, D, V, [(1, at, c)], state, decay, table, rot, ks, dt))
            at += c
        assert rel_err(torch.cat(outs), ref) < 2e-5, cuts
        assert rel_err(state[1], S_ref) < 2e-5
        assert float(state[2].abs().max()) == 0.0


@pytest.mark.parametrize("kind,dt", [("scan", F32), ("scan", BF16), ("chunks", BF16)])
def test_retention_in_a_mixed_batch_of_continuations(kind, dt):
    from builderforce_inference_b200.parts.rotary import rotary_table
    H, D, V, rot, base = 2, 32, 48, 32, 1e3
    g = torch.Generator().manual_seed(8)
    decay, table = torch.tensor([0.9, 0.999]), rotary_table(base, rot, 1024, DEV)
    seqs = [(4, 0, 128), (0, 37, 65), (2, 900, 1), (1, 64, 63), (3, 5, 2)]
    start = 0.3 * torch.randn(5, H, D, V, generator=g)
    state = start.clone().to(DEV)
    proj = torch.randn(sum(t for _, _, t in seqs), 2 * H * D + H * V, generator=g)
    got, at = run_retention(kind, proj, H, D, V, seqs, state, decay, table, rot, 0.2, dt), 0
    for slot, st, t in seqs:
        ref, S_end = plain_retention(proj[at:at + t], H, D, V, decay, st, rot, base, 0.2, dt, start[slot].double())
        assert rel_err(got[at:at + t], ref) < 2e-5 and rel_err(state[slot], S_end) < 2e-5
        at += t


@pytest.mark.parametrize("kind,dt", [("scan", F32), ("scan", BF16), ("chunks", BF16)])
def test_retention_answers_one_loud_key_by_its_distance(kind, dt):
    """One key and value among silent ones: every later output is its value times decay^distance times
    (q rotated at t) . (k rotated at its place), which depends on the distance alone, also 500 tokens on and
    over steps; earlier outputs and the other head stay silent."""
    from builderforce_inference_b200.parts.rotary import rotary_table
    H, D, V, rot, base, n, loud = 2, 32, 16, 32, 1e4, 600, 70
    decay, table = torch.tensor([0.999, 0.5]), rotary_table(base, rot, 1024, DEV)
    proj = torch.zeros(n, 2 * H * D + H * V)
    proj[:, :D] = 1.0                                     # every query of head 0
    proj[loud, H * D:H * D + D] = 2.0                     # one key
    proj[loud, 2 * H * D:2 * H * D + V] = 3.0             # and its value
    i = torch.arange(rot // 2, dtype=P.F)
    freq = base ** (-2.0 * i / rot)
    for cuts in ([n], [60, 5, 300, 235], [loud + 1] + [1] * 9 + [n - loud - 10]):
        state, outs, at = torch.zeros(1, H, D, V, dtype=F32, device=DEV), [], 0
        for c in cuts:
            outs.append(run_retention(kind if c > 1 else "scan", proj[at:at + c], H, D, V, [(0, at, c)], state, decay, table, rot, 0.5, dt))
            at += c
        got = torch.cat(outs)
        assert float(got[:loud].abs().max()) == 0.0 and float(got[:, V:].abs().max()) == 0.0
        for t in (loud, loud + 1, loud + 63, loud + 64, 255, 256, n - 1):
            want = 3.0 * float(decay[0].double()) ** (t - loud) * float((2.0 * torch.cos((t - loud) * freq)).sum()) * 2.0 * 0.5
            assert abs(float(got[t, 0]) - want) < 2e-3 * 32, (cuts, t)


def test_a_position_outside_the_rotation_table_is_recorded():
    from builderforce_inference_b200.parts.rotary import rotary_table
    o = ops()
    table, status = rotary_table(10.0, 8, 16, DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    out, state = torch.zeros(1, 8, device=DEV), torch.zeros(1, 1, 8, 8, device=DEV)
    o.lightning_scan(torch.randn(1, 24, device=DEV), 0, 8, 16, out, state, torch.ones(1, device=DEV), i32([0, 1]), i32([0]), 1, 1, 8, 8,
                     o.LIGHT_ACT_NONE, single_tokens=True, rope_table=table, rot_dim=8, token_pos=i32([16]), status=status)
    assert int(status) == o.STATUS_BAD_POSITION


@pytest.mark.parametrize("dt", [F32, BF16])
def test_norm_per_head_without_weight_and_silu_gate(dt):
    o = ops()
    g = torch.Generator().manual_seed(8)
    for n, H, V in ((5, 3, 7), (9, 1, 64), (2, 16, 128)):
        x = torch.randn(n, H * V, generator=g) * torch.logspace(-4, 1, n)[:, None]       # down to where eps matters
        gate = 2.0 * torch.randn(n, H * V + 5, generator=g)
        y = torch.empty(n, H * V, dtype=dt, device=DEV)
        o.gated_group_norm(x.to(DEV), gate.to(dt).to(DEV)[:, 2:2 + H * V], None, 1e-5, y, H, gate_first=False, gate_act=o.GATE_SILU)
        z = q64(gate, dt)[:, 2:2 + H * V]
        ref = P.rms(x.double().view(n, H, V), 1e-5).reshape(n, H * V) * z * torch.sigmoid(z)
        assert rel_err(y, ref) < (1e-6 if dt == F32 else 8e-3)


# ------------------------------------------------------------------------------------------------
# feed-forwards, soft cap
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n_rows", [1, 3, 8, 40, 70, 127, 128, 300])
@pytest.mark.parametrize("n,k", [(36, 40), (200, 64), (385, 256), (2048, 512), (20, 35)])
def test_products_that_square_the_relu(dt, n_rows, n, k):
    from builderforce_inference_b200.kernels.linear import EPI_RELU_SQUARED, linear
    g = torch.Generator().manual_seed(n + k)
    a, w = torch.randn(n_rows, k, generator=g), torch.randn(n, k, generator=g) / math.sqrt(k)
    for out_dt in {dt, F32}:
        out = torch.full((n_rows, n), float("nan"), dtype=out_dt, device=DEV)
        linear(a.to(dt).to(DEV), w.to(dt).to(DEV), out, EPI_RELU_SQUARED)
        ref = torch.clamp(q64(a, dt) @ q64(w, dt).T, min=0.0) ** 2
        assert rel_err(out, ref) < (1e-5 if out_dt == F32 else 6e-3)
        assert float(out[ref.to(DEV) == 0.0].float().abs().max()) < 1e-9


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n_rows", [1, 3, 8, 40, 70, 127, 128, 300])
@pytest.mark.parametrize("E,ff,k", [(5, 20, 40), (8, 64, 128), (3, 7, 64), (16, 48, 512), (1, 33, 35)])
def test_gated_products_with_factors_on_their_input(dt, n_rows, E, ff, k):
    """Row m and expert e share a factor on gate and up, before clamp and activation; a factor of 0 leaves
    exactly 0."""
    from builderforce_inference_b200.kernels.linear import EPI_SWIGLU, linear
    g = torch.Generator().manual_seed(E + ff)
    a = torch.randn(n_rows, k, generator=g)
    wg, wu = (torch.randn(E * ff, k, generator=g) / math.sqrt(k) for _ in range(2))
    f = torch.rand(n_rows, E, generator=g) * (torch.rand(n_rows, E, generator=g) < 0.6)
    w = torch.stack([wg, wu], dim=1).reshape(2 * E * ff, k)
    out = torch.full((n_rows, E * ff), float("nan"), dtype=dt, device=DEV)
    linear(a.to(dt).to(DEV), w.to(dt).to(DEV), out, EPI_SWIGLU, (1.702, 0.7, 1.0), in_scale=(f.to(DEV), ff))
    fx = f.double().repeat_interleave(ff, dim=1)
    gate = torch.clamp(q64(a, dt) @ q64(wg, dt).T * fx, max=0.7)
    up = torch.clamp(q64(a, dt) @ q64(wu, dt).T * fx, min=-0.7, max=0.7)
    ref = gate * torch.sigmoid(1.702 * gate) * (up + 1.0)
    assert rel_err(out, ref) < (1e-5 if dt == F32 else 6e-3)
    assert torch.equal(out.cpu() == 0, (fx == 0) | (out.cpu() == 0))
    # the factors belong to that one product: the next one has none
    plain = torch.empty_like(out)
    linear(a.to(dt).to(DEV), w.to(dt).to(DEV), plain, EPI_SWIGLU)
    z = q64(a, dt) @ q64(wg, dt).T
    assert rel_err(plain, z * torch.sigmoid(z) * (q64(a, dt) @ q64(wu, dt).T)) < (1e-5 if dt == F32 else 8e-3)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("E,top,ff,width,limit", [(5, 3, 20, 40, 0.5), (8, 1, 64, 128, 1.0), (1, 1, 7, 33, 0.3), (12, 4, 32, 256, 7.0)])
@pytest.mark.parametrize("n", [1, 4, 30, 200])
def test_routed_feed_forward_with_weights_on_the_input(dt, E, top, ff, width, limit, n):
    """Both ways of computing (chosen experts; every expert with factor 0 for those not chosen, in steps of
    enough tokens) against the plain routed feed-forward, with routers that decide by the scores."""
    from builderforce_inference_b200.engine.context import Workspace, build_context
    from builderforce_inference_b200.engine.decoder import Runtime
    from builderforce_inference_b200.parts.base import FEED_FORWARDS, PartSpec
    part = FEED_FORWARDS.build(PartSpec("mixture_of_experts", {
        "width": width, "n_experts": E, "top": top, "inner": ff, "correction": False, "score": "sigmoid", "gate_alpha": 1.702, "limit": limit,
        "up_shift": 1.0, "weight_on": "input"}))
    g = torch.Generator().manual_seed(E * ff + n)
    w = {"router": torch.randn(E, width, generator=g) * (2.0 / math.sqrt(width))}
    for e in range(E):
        for kind, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            w[f"e{e}.{kind}"] = torch.randn(shape, generator=g) * (1.5 / math.sqrt(shape[1]))
    part.load_all({("router" if k == "router" else f"experts.{k[1:].replace('.', '.')}_proj"): v.to(dt).to(DEV) for k, v in w.items()}, Runtime(DEV, dt))
    h = torch.randn(n, width, generator=g)
    w64 = {k: q64(v, dt) for k, v in w.items()}
    rep = []
    ref = P.routed_ff(q64(h, dt), w64, "", {"router": {"experts": E, "top": top}, "expert": {"limit": limit}}, rep)
    assert not rep or min(rep) > 1e-6
    ctx = build_context([(0, 0, [0] * n)], dt, Workspace(DEV), DEV)
    out = torch.full((n, width), float("nan"), device=DEV)
    part.forward_store(ctx, h.to(dt).to(DEV), out)
    assert rel_err(out, ref) < (1e-5 if dt == F32 else 1.5e-2)
    acc = torch.ones(n, width, device=DEV)
    part.forward(ctx, h.to(dt).to(DEV), acc)
    assert rel_err(acc - 1.0, out) < 1e-5


def test_router_writes_every_experts_weight():
    o = ops()
    g = torch.Generator().manual_seed(3)
    n, E, top, width = 40, 9, 2, 48
    h, wr = torch.randn(n, width, generator=g), torch.randn(E, width, generator=g) * 0.3
    slots = [0] * n
    slots[7] = -1
    idx, wt = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
    every = torch.full((n, E), float("nan"), device=DEV)
    o.moe_router(h.to(DEV), wr.to(DEV), E, None, i32(slots), idx, wt, top, score=o.SCORE_SIGMOID, dense_weight=every)
    ridx, rw = P.route(h.double(), wr.double(), top)
    want = torch.zeros(n, E, dtype=P.F).scatter_(1, ridx, rw)
    want[7] = 0.0                                          # a padding row
    assert rel_err(every, want) < 1e-6


def test_soft_cap():
    g = torch.Generator().manual_seed(1)
    big = torch.randn(3, 700, generator=g) * torch.tensor([[0.01], [5.0], [300.0]])
    x = big.to(DEV)
    ops().softcap_rows(x[:, :613], 4.0)
    assert rel_err(x[:, :613], 4.0 * torch.tanh(big[:, :613].double() / 4.0)) < 1e-6
    assert torch.equal(x[:, 613:].cpu(), big[:, 613:])
    small = 4.0 * torch.tanh(big[0, :613].double() / 4.0)
    assert rel_err(x[0, :613], small) < 1e-6


@pytest.mark.parametrize("width", [512, 1028, 2560, 8192])
@pytest.mark.parametrize("dt", [F32, BF16])
def test_normed_add_with_the_next_norm_over_wide_rows(width, dt):
    """Rows of a served model's width take the kernel that keeps a row in registers: few rows and many, with
    and without the norm that follows, weights of either storage type."""
    o = ops()
    g = torch.Generator().manual_seed(width)
    for n in (3, 400):
        x, y = torch.randn(n, width, generator=g), 0.2 * torch.randn(n, width, generator=g)
        w, w2 = (1.0 + 0.2 * torch.randn(width, generator=g) for _ in range(2))
        ref = x.double() + P.rms(y.double(), 1e-5) * q64(w, dt)
        xd, h = x.to(DEV), torch.full((n, width), float("nan"), dtype=dt, device=DEV)
        o.norm_add(xd, y.to(DEV), w.to(dt).to(DEV), 1e-5, next_w=w2.to(DEV), next_eps=1e-6, out=h)
        assert rel_err(xd, ref) < 1e-6
        assert rel_err(h, P.rms(ref, 1e-6) * w2.double()) < (1e-6 if dt == F32 else 8e-3)
        xd = x.to(DEV)
        o.norm_add(xd, y.to(DEV), w.to(dt).to(DEV), 1e-5)
        assert rel_err(xd, ref) < 1e-6


# ------------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_whole_prompts_and_every_layer(name, dtype):
    from builderforce_inference_b200.engine.context import build_context
    eng, cfg, w = engine(name, dtype)
    ids = prompts(cfg["vocab"], [330])[0]
    layers = []
    ref = P.forward(cfg, w, ids, layers)
    slot = eng.acquire()
    assert close(eng.step([S(slot, ids)]), ref, dtype)
    eng.release(slot)
    # the residual stream after every layer
    slot = eng.acquire()
    eng.cache.begin_step([slot], [len(ids)])
    ctx = build_context([(slot, 0, ids)], eng.dtype, eng.workspace, eng.device, eng.status)
    x = eng.decoder.embed(ctx)
    for i in range(len(cfg["layers"])):
        eng.decoder.run_layers(ctx, x, eng.cache, i, i + 1)
        assert close(x, layers[i], dtype), i
    eng.cache.end_step([slot], [len(ids)])
    eng.release(slot)
    eng.cache.check()
    eng.check_status()


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_prompt_then_token_by_token_far_past_every_window(name, dtype, graphs):
    eng, cfg, w = engine(name, dtype, use_graphs=graphs)
    ids = prompts(cfg["vocab"], [330], 40)[0]              # windows of 9 to 130 positions pass over decoded tokens
    ref = P.forward(cfg, w, ids)
    slot = eng.acquire()
    head = 3
    outs = [eng.step([S(slot, ids[:head])]).clone()]
    for t in ids[head:]:
        outs.append(eng.step([S(slot, [t])]).clone())
    assert close(torch.cat(outs), ref, dtype)
    for gkv in eng.cache.kv_groups:                        # the first positions' pages and the window's, no others
        held = sum(1 for p in gkv.table.rows[slot] if p >= 0)
        assert held <= (gkv.need.window + 62) // 64 + 1 + (gkv.need.keep_first + 63) // 64
    eng.release(slot)
    eng.cache.check()
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_portions_of_a_prompt_down_to_two_tokens(name, dtype):
    eng, cfg, w = engine(name, dtype)
    ids = prompts(cfg["vocab"], [331], 70)[0]
    ref = P.forward(cfg, w, ids)
    for cuts in ([2, 2, 3, 64, 65, 63, 2, 130], [128, 203], [1, 7, 1, 130, 192], [1, 330], [2] * 165 + [1]):
        slot = eng.acquire()
        outs, at = [], 0
        for c in cuts:
            outs.append(eng.step([S(slot, ids[at:at + c])]).clone())
            at += c
        assert at == len(ids)
        assert close(torch.cat(outs), ref, dtype), cuts
        eng.release(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_step_cut_into_micro_batches(dtype):
    eng, cfg, w = engine("wide", dtype, prefill_chunk_tokens=128)
    seqs = prompts(cfg["vocab"], [300, 7, 141], 12)
    slots = [eng.acquire() for _ in seqs]
    got = eng.step([S(sl, s) for sl, s in zip(slots, seqs)])
    assert close(got, torch.cat([P.forward(cfg, w, s) for s in seqs]), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_unequal_batches_reused_slots_and_poisoned_pages(name, dtype):
    eng, cfg, w = engine(name, dtype, max_tokens=1024)
    eng.cache.poison()
    lengths = [70, 5, 211, 1]
    seqs = [prompts(cfg["vocab"], [n + 6], 100 + i)[0] for i, n in enumerate(lengths)]
    refs = [P.forward(cfg, w, s) for s in seqs]
    for round_ in range(2):                               # the second round runs in slots and pages that were used
        slots = [eng.acquire() for _ in seqs]
        got = eng.step([S(sl, s[:n]) for sl, s, n in zip(slots, seqs, lengths)])
        want = torch.cat([r[:n] for r, n in zip(refs, lengths)])
        assert close(got, want, dtype), round_
        live = list(range(len(seqs)))
        for step in range(6):                             # decoded together; the shortest leave first
            got = eng.step([S(slots[i], [seqs[i][lengths[i] + step]]) for i in live])
            want = torch.stack([refs[i][lengths[i] + step] for i in live])
            assert close(got, want, dtype), (round_, step)
            if step in (1, 3):
                eng.release(slots[live.pop(1)])
        for i in live:
            eng.release(slots[i])
        eng.cache.check()
        eng.cache.poison()


@pytest.mark.parametrize("name", ["odd", "wide"])
def test_batch_against_each_alone_in_float32(name):
    eng, cfg, w = engine(name, "float32")
    seqs = prompts(cfg["vocab"], [33, 240, 2, 71], seed=9)
    slots = [eng.acquire() for _ in seqs]
    together = eng.step([S(sl, s) for sl, s in zip(slots, seqs)]).clone()
    nxt = eng.step([S(sl, [7]) for sl in slots]).clone()
    for sl in slots:
        eng.release(sl)
    at = 0
    for i, s in enumerate(seqs):
        sl = eng.acquire()
        alone = eng.step([S(sl, s)]).clone()
        # the products' tiles differ with the number of rows, so sums differ in their last bits
        assert rel_err(together[at:at + len(s)], alone) < 1e-5
        assert rel_err(nxt[i:i + 1], eng.step([S(sl, [7])])) < 1e-5
        eng.release(sl)
        at += len(s)


@pytest.mark.parametrize("seed", range(101, 125))
def test_random_configurations_in_float32(seed):
    """Configurations drawn from a seed (layer order, every size, masks, borrowed keys, rotation, routers,
    with and without feed-forward): an unequal batch of prompts, five tokens decoded together, and the
    longest prompt again in portions, against the plain implementation.  A prompt whose routers decide by
    less than 1e-4 somewhere is not compared (a float32 sum may turn it)."""
    from builderforce_inference_b200.engine.engine import Engine
    cfg = random_config(seed)
    w = make_weights(cfg, seed, F32)
    eng = Engine.load(write_folder(cfg, w), dtype="float32", max_tokens=2048)
    w64 = {k: v.to(torch.float64) for k, v in w.items()}
    lens = [(1, 5, 70, 130, 260)[seed % 5], (2, 33, 200)[seed % 3], (1, 64, 129)[seed % 2]]
    seqs = prompts(cfg["vocab"], [n + 5 for n in lens], seed)
    refs, steady = [], []
    for s in seqs:
        rep = []
        refs.append(P.forward(cfg, w64, s, None, rep))
        steady.append(not rep or min(rep) > 1e-4)
    slots = [eng.acquire() for _ in seqs]
    got = eng.step([S(sl, s[:n]) for sl, s, n in zip(slots, seqs, lens)])
    at = 0
    for i, n in enumerate(lens):
        if steady[i]:
            assert rel_err(got[at:at + n], refs[i][:n]) < 4e-4, (i, cfg)
        at += n
    for step in range(5):
        got = eng.step([S(sl, [s[n + step]]) for sl, s, n in zip(slots, seqs, lens)])
        for i, n in enumerate(lens):
            if steady[i]:
                assert rel_err(got[i:i + 1], refs[i][n + step:n + step + 1]) < 4e-4, (i, step, cfg)
    for sl in slots:
        eng.release(sl)
    i = max(range(3), key=lambda k: lens[k])
    sl, outs, at = eng.acquire(), [], 0
    for c in [max(1, lens[i] // 3), 2, 1, 97, 10 ** 6]:
        c = min(c, lens[i] - at)
        if c > 0:
            outs.append(eng.step([S(sl, seqs[i][at:at + c])]).clone())
            at += c
    if steady[i]:
        assert rel_err(torch.cat(outs), refs[i][:lens[i]]) < 4e-4, cfg
    eng.release(sl)
    eng.cache.check()
    eng.check_status()


@pytest.mark.parametrize("seed", range(201, 213))
def test_random_configurations_in_bfloat16(seed):
    """The same draw in bfloat16 with experts that resemble one another: a prompt whole, in portions and
    its end token by token stay close to the plain implementation."""
    from builderforce_inference_b200.engine.engine import Engine
    cfg = random_config(seed)
    w = make_weights(cfg, seed, BF16, steady=True)
    eng = Engine.load(write_folder(cfg, w), dtype="bfloat16", max_tokens=1024)
    ids = prompts(cfg["vocab"], [230], seed)[0]
    ref = P.forward(cfg, {k: v.to(torch.float64) for k, v in w.items()}, ids)
    for cuts in ([230], [150, 70] + [1] * 10):
        sl, outs, at = eng.acquire(), [], 0
        for c in cuts:
            outs.append(eng.step([S(sl, ids[at:at + c])]).clone())
            at += c
        # among a few hundred tokens of a random model some are badly conditioned; most rows must be right
        err = (torch.cat(outs).double().cpu() - ref).abs().max(dim=1).values / float(ref.abs().max())
        assert float(err.median()) < 8e-2 and float(err.quantile(0.9)) < 0.25, (cuts, cfg)
        eng.release(sl)


@pytest.mark.parametrize("name", ["odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_public_entry_point(name, dtype):
    from builderforce_inference_b200.engine.api import Model
    from builderforce_inference_b200.sampling.params import SampleParams
    folder, cfg, w = model(name, dtype)
    m = Model.load(folder, dtype=dtype, max_tokens=1024)
    ps = prompts(cfg["vocab"], [12, 3, 140], seed=21)
    n_new = 24
    outs = m.generate_batch(ps, SampleParams(temperature=0.0, max_tokens=n_new), ignore_eos=True)
    for p, got in zip(ps, outs):
        got = list(got)
        assert len(got) == n_new
        # every generated id is the plain model's best id given the ids before it, or (bfloat16) a near tie
        ref = P.forward(cfg, w, p + got)
        for i, tok in enumerate(got):
            row = ref[len(p) + i - 1]
            if int(torch.argmax(row)) != tok:
                assert dtype == "bfloat16" and float(row.max() - row[tok]) < 0.08 * float(row.max() - row.min())


def test_random_weights_and_a_byte_budget_take_the_design():
    """``from_random`` and the cache's byte plan know the design (the command line's two ways in)."""
    from builderforce_inference_b200.engine.engine import Engine
    from zirivik_models import ZV_ODD
    eng = Engine.from_random(ZV_ODD, 5, dtype="bfloat16", cache_bytes=1 << 24, cache_slots=4)
    assert eng.cache_plan.n_slots == 4 and eng.cache_plan.state_bytes_per_slot == 4 * (3 * 10 * 6 + 2 * 24 * 40)
    sl = eng.acquire()
    assert torch.isfinite(eng.step([S(sl, [1, 2, 3])])).all()


def test_trace_replay_takes_the_model():
    import subprocess
    import sys
    import tempfile

    import numpy as np

    from helpers import ROOT
    folder, cfg, w = model("odd", "float32")
    a, b = prompts(cfg["vocab"], [140, 9], seed=31)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:130], "want": [0, 129]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[130:131], "want": [0]}, {"id": "b", "tokens": b[8:9], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[131:140], "want": [8]}], "end": ["a"]}]
    out_dir = tempfile.mkdtemp(prefix="bfi_trace_")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", out_dir,
                        "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                       timeout=900)
    assert r.returncode == 0, r.stderr[-3000:]
    assert [line for line in r.stdout.splitlines() if line.startswith("done ")] == ["done 0", "done 1", "done 2"]
    ra, rb = P.forward(cfg, w, a), P.forward(cfg, w, b)
    for step, want in ((0, torch.stack([ra[0], ra[129], rb[7]])), (1, ra[130:131]), (2, ra[139:140])):
        got = torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{step}.f32"), dtype="<f4").reshape(want.shape[0], -1).copy())
        assert rel_err(got, want) < 3e-5

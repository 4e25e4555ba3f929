"""Zitezen through the package against the plain implementation (tests/plain/zitezen_plain.py): every
mechanism's kernel alone, then whole models with sizes of their own, stepped whole, token by token,
in portions, in unequal batches, over reused slots and pages, and generated from greedily.

Some tests shape their inputs so that one key, one gate or one copy decides the result."""
import json
import math
import os

import pytest
import torch

from attention_pages import Pages
from helpers import rel_err
from plain import zitezen_plain as P
from zitezen_models import BF16, F32, make_weights, model, prompts, random_config, write_folder

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")


def close(got, ref, dtype):
    """Whether a model's output is the plain implementation's.  float32: every value, to 3e-5 of the
    largest.  bfloat16: 95 % of the rows (all but one, of few) lie within 6e-2 and every row is finite and
    within 1, since rounding is amplified where a token is badly conditioned; a lost state or a wrong key
    shows as 0.3 and more.  The float32 run is the sharp test."""
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
# the copies of the residual stream and the norm without statistics
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("width", [42, 64, 1028])
@pytest.mark.parametrize("s", [1, 2, 3, 4, 5, 8, 32])
def test_dynamic_tanh_of_the_copies(dt, width, s):
    o = ops()
    g = torch.Generator().manual_seed(width + s)
    n = 7
    x, read = torch.randn(n, s * width, generator=g), torch.randn(s, generator=g)
    alpha, w, b = torch.tensor([0.7]), torch.randn(width, generator=g), torch.randn(width, generator=g)
    X = x.double().view(n, s, width)
    norm = (alpha.to(DEV), w.to(dt).to(DEV), b.to(dt).to(DEV))
    for rows in (None, [6, 0, 0, 3]):
        pick = X if rows is None else X[rows]
        for weights in (read, None):
            u = torch.einsum("a,taw->tw", read.double() if weights is not None else torch.ones(s, dtype=P.F), pick)
            ref = P.dynamic_tanh(u, 0.7, q64(w, dt), q64(b, dt))
            out = torch.full((u.shape[0], width), float("nan"), dtype=dt, device=DEV)
            u_out = torch.full((u.shape[0], width), float("nan"), device=DEV)
            o.dynamic_tanh(x.to(DEV), out, *norm, rows=None if rows is None else i32(rows), streams=s,
                           read=None if weights is None else read.to(DEV), u_out=u_out)
            assert rel_err(u_out, u) < 2e-6 and rel_err(out, ref) < (3e-6 if dt == F32 else 5e-3)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("width", [42, 64, 1028])
@pytest.mark.parametrize("s", [1, 2, 3, 4, 5, 8, 32])
def test_a_sublayers_output_into_the_copies(dt, width, s):
    """All copies from the old ones, the matrix indexed [from, to]; one term or two with factors, with and
    without a scale per channel; what the next sublayer reads comes from the new copies."""
    o = ops()
    g = torch.Generator().manual_seed(width * 7 + s)
    n = 5
    x, y0, y1 = (torch.randn(n, c, generator=g) for c in (s * width, width, width))
    mix, write, read = torch.randn(s, s, generator=g) / math.sqrt(s), torch.randn(s, generator=g), torch.randn(s, generator=g)
    scale, w, b = (torch.randn(width, generator=g) for _ in range(3))
    alpha = torch.tensor([0.4])
    for terms, ref_y, sc in (([(y0, 1.0)], y0.double(), None), ([(y0, 0.8)], 0.8 * y0.double(), scale),
                             ([(y0, 0.6), (y1, -1.3)], 0.6 * y0.double() - 1.3 * y1.double(), scale)):
        ref_y = ref_y if sc is None else ref_y * q64(sc, dt)
        want = P.connect(x.double().view(n, s, width).permute(1, 0, 2), torch.zeros(s, dtype=P.F), write.double(), mix.double(), lambda u: ref_y)
        u = torch.einsum("a,atw->tw", read.double(), want)
        for follow in ("nothing", "sum", "norm", "both"):
            xd = x.to(DEV)
            h = torch.full((n, width), float("nan"), dtype=dt, device=DEV) if follow in ("norm", "both") else None
            uo = torch.full((n, width), float("nan"), device=DEV) if follow in ("sum", "both") else None
            o.stream_mix(xd, s, [(y.to(DEV), c) for y, c in terms], None if sc is None else sc.to(dt).to(DEV), mix.to(DEV), write.to(DEV),
                         read=None if follow == "nothing" else read.to(DEV),
                         norm=None if h is None else (alpha.to(DEV), w.to(dt).to(DEV), b.to(dt).to(DEV)), out=h, u_out=uo)
            assert rel_err(xd.view(n, s, width), want.permute(1, 0, 2)) < 2e-6
            if uo is not None:
                assert rel_err(uo, u) < 4e-6
            if h is not None:
                assert rel_err(h, P.dynamic_tanh(u, 0.4, q64(w, dt), q64(b, dt))) < (4e-6 if dt == F32 else 5e-3)


def test_the_tanh_keeps_its_ends():
    """Far out the norm is exactly b + w or b - w, near zero it is alpha * x * w + b, with a small alpha and
    a large one."""
    o = ops()
    x = torch.tensor([[-1e6, -40.0, -1e-4, 0.0, 1e-4, 40.0, 1e6, float("inf")]])
    for alpha in (0.01, 3.0):
        out = torch.empty(1, 8, device=DEV)
        o.dynamic_tanh(x.to(DEV), out, torch.tensor([alpha], device=DEV), torch.full((8,), 2.0, device=DEV), torch.zeros(8, device=DEV))
        assert rel_err(out, 2.0 * torch.tanh(alpha * x.double())) < 1e-6
        assert abs(float(out[0, 4]) / (2e-4 * alpha) - 1.0) < 1e-5 and float(out[0, 7]) == 2.0


# ------------------------------------------------------------------------------------------------
# soft-capped attention
# ------------------------------------------------------------------------------------------------
def capped(q, k, v, scale, cap, dt):
    group = q.shape[1] // k.shape[1]
    return P.causal_attention(q64(q, dt), q64(k, dt).repeat_interleave(group, dim=1), q64(v, dt).repeat_interleave(group, dim=1), scale,
                              cap).reshape(q.shape[0], -1)


def attend(kind, q, pages, seqs, n_q, dv, scale, cap, dt):
    """One step through the kernel ``kind``: "general", "decode", "short" (mma.sync prompt kernel), "long"
    (tcgen05), or "chosen", the one the attention part takes."""
    from builderforce_inference_b200.engine.context import Workspace, build_context
    from builderforce_inference_b200.kernels import attention as choose
    from builderforce_inference_b200.kernels import fast_ops
    ctx = build_context([(s, st, [0] * t) for s, st, t in seqs], dt, Workspace(DEV), DEV)
    qd = q.to(dt).to(DEV).contiguous()
    out = torch.full((qd.shape[0], n_q * dv), float("nan"), dtype=dt, device=DEV)
    if kind == "general":
        ops().attention_paged(qd, qd.stride(0), out, pages.view, ctx.cu_seqlens, ctx.seq_slot, ctx.seq_start, ctx.n_seqs,
                              ctx.max_seq_tokens, n_q, scale, softcap=cap)
    elif kind == "decode":
        assert fast_ops.attention_decode_bf16(ctx, qd, out, pages.view, n_q, scale, exact_weights=True, softcap=cap)
    elif kind == "short":
        assert fast_ops.attention_prefill_bf16(ctx, qd, out, pages.view, n_q, scale, None, True, cap)
    elif kind == "long":
        assert fast_ops.attention_prefill_tcgen05_bf16(ctx, qd, out, pages.view, n_q, scale, None, True, cap)
    else:
        assert choose.attend(ctx, qd, out, pages.view, n_q, scale, None, True, cap)
    if kind in ("decode", "long", "chosen"):
        assert int(fast_ops.tc_status(DEV)[0]) == 0
    return out.double().cpu()


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n_q,n_kv,d,dv", [(4, 2, 24, 10), (6, 1, 16, 40), (3, 3, 48, 48)])
@pytest.mark.parametrize("cap", [0.4, 5.0, 40.0])
def test_general_attention_caps_its_scores_in_a_mixed_batch(dt, n_q, n_kv, d, dv, cap):
    g = torch.Generator().manual_seed(n_q * 100 + d)
    seqs = [(2, 0, 150), (0, 330, 1), (1, 261, 7), (3, 0, 2)]
    pages = Pages(4, 384, n_kv, d, dv, dt, None, 0)
    qs, refs = [], []
    for slot, start, t in seqs:
        n = start + t
        k, v, q = (3.0 * torch.randn(n, h, e, generator=g) for h, e in ((n_kv, d), (n_kv, dv), (n_q, d)))
        pages.write(slot, k, v)
        refs.append(capped(q, k, v, 0.2, cap, dt)[start:])
        qs.append(q[start:].reshape(t, n_q * d))
    got = attend("general", torch.cat(qs), pages, seqs, n_q, dv, 0.2, cap, dt)
    assert rel_err(got, torch.cat(refs)) < (5e-6 if dt == F32 else 1e-2)


@pytest.mark.parametrize("n_q,n_kv,d", [(8, 2, 64), (4, 1, 128), (40, 2, 64), (2, 2, 128)])
@pytest.mark.parametrize("cap", [0.4, 5.0, 40.0])
def test_tensor_core_attention_caps_its_scores(n_q, n_kv, d, cap):
    """The three bfloat16 kernels in unequal batches.  The weights are float32 in effect, so what is left
    is the rounding of the output."""
    g = torch.Generator().manual_seed(n_q + d)
    lens = [700, 131, 1, 449]
    pages = Pages(4, 704, n_kv, d, d, BF16, None, 0)
    data = []
    for slot, n in enumerate(lens):
        k, v, q = (3.0 * torch.randn(n, h, d, generator=g) for h in (n_kv, n_kv, n_q))
        pages.write(slot, k, v)
        data.append((q, capped(q, k, v, 0.15, cap, BF16)))

    def check(kind, seqs):
        got = attend(kind, torch.cat([data[s][0][st:st + t] for s, st, t in seqs]).reshape(-1, n_q * d), pages, seqs, n_q, d, 0.15, cap, BF16)
        ref = torch.cat([data[s][1][st:st + t] for s, st, t in seqs])
        step = 2.0 ** (math.floor(math.log2(float(ref.abs().max()))) - 7)       # of bfloat16 at the largest output
        assert float((got - ref.to(BF16).double()).abs().max()) <= step, (kind, seqs)

    for kind in ("long", "short", "chosen"):
        check(kind, [(1, 0, 131), (0, 0, 700), (2, 0, 1), (3, 0, 449)])
        check(kind, [(0, 500, 200), (1, 129, 2), (3, 65, 384)])
    for kind in ("decode", "chosen"):
        check(kind, [(0, 699, 1), (1, 130, 1), (2, 0, 1), (3, 448, 1)])
        check(kind, [(3, 64, 1), (1, 63, 1), (0, 9, 1)])


@pytest.mark.parametrize("kind,dt,d", [("general", F32, 16), ("general", BF16, 16), ("decode", BF16, 64), ("short", BF16, 64), ("long", BF16, 64),
                                       ("decode", BF16, 128), ("short", BF16, 128), ("long", BF16, 128)])
@pytest.mark.parametrize("cap", [3.0, 12.0])
def test_one_loud_key_is_heard_as_loud_as_its_cap(kind, dt, d, cap):
    """Among quiet keys one has a score far above the cap: it weighs e^cap against the others' e^0, wherever
    it lies and however far back, in a prompt, in a portion of one and as a single decoded token."""
    n_q, n_kv, n = 2, 1, 400
    g = torch.Generator().manual_seed(int(cap))
    for loud in (0, 1, 63, 64, 200, 255):
        k, v, q = (torch.zeros(n, h, d) for h in (n_kv, n_kv, n_q))
        v[:, 0, 1:] = torch.randn(n, d - 1, generator=g)
        k[loud, 0, 0], q[:, :, 0], v[loud, 0, 0] = 40.0, 40.0, 8.0
        pages = Pages(1, n, n_kv, d, d, dt, None, 0, seed=loud)
        pages.write(0, k, v)
        ref = capped(q, k, v, 0.25, cap, dt)
        spots = sorted({loud, loud + 1, 64, 319, 320, n - 1})
        runs = [(p, 1) for p in spots if p >= loud] if kind == "decode" else \
            [(0, n)] + [(p, min(n - p, c)) for p in spots for c in (2, 130) if loud <= p < n - 1]
        for start, t in runs:
            got = attend(kind, q[start:start + t].reshape(t, -1), pages, [(0, start, t)], n_q, d, 0.25, cap, dt)
            assert rel_err(got, ref[start:start + t]) < (1e-5 if dt == F32 else 1e-2), (loud, start, t)
            for i in range(t):
                p = start + i
                want = 0.0 if p < loud else 8.0 * math.exp(cap) / (math.exp(cap) + p)
                assert abs(float(got[i, 0]) - want) < 0.05, (loud, p)


def test_the_cap_goes_with_a_window_and_kept_first_positions():
    n_q, n_kv, d, n, window, keep, cap = 4, 2, 64, 300, 70, 5, 2.0
    g = torch.Generator().manual_seed(3)
    k, v, q = (2.0 * torch.randn(n, h, d, generator=g) for h in (n_kv, n_kv, n_q))
    s = P.soft_cap(torch.einsum("iad,jad->aij", q64(q, BF16), q64(k, BF16).repeat_interleave(2, dim=1)) * 0.2, cap)
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = (j <= i) & ((i - j < window) | (j < keep))
    w = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)
    ref = torch.einsum("aij,jad->iad", w, q64(v, BF16).repeat_interleave(2, dim=1)).reshape(n, -1)
    pages = Pages(1, n, n_kv, d, d, BF16, window, keep)
    pages.write(0, k, v)
    for kind, runs in (("general", [(0, n), (200, 1)]), ("short", [(0, n), (100, 130)]), ("long", [(0, n), (100, 130)]), ("decode", [(299, 1), (72, 1)])):
        for start, t in runs:
            got = attend(kind, q[start:start + t].reshape(t, -1), pages, [(0, start, t)], n_q, d, 0.2, cap, BF16)
            assert rel_err(got, ref[start:start + t]) < 1e-2, (kind, start)


# ------------------------------------------------------------------------------------------------
# the matrix memory
# ------------------------------------------------------------------------------------------------
class Memory:
    """Inputs of one memory layer for the kernels and the plain scan: projections ``[T, q | k | v]`` behind a
    few unused columns, the layer's input and gate rows (or gate logits, where a test sets them itself)."""

    def __init__(self, H, D, V, n, dt, width=40, cap=9.0, seed=0, zi=None, zf=None):
        g = torch.Generator().manual_seed(seed + H * D + V)
        self.H, self.D, self.V, self.dt, self.cap, self.n = H, D, V, dt, cap, n
        up = lambda x: (x + 7) // 8 * 8
        self.q_off, self.k_off, self.v_off = 8, 8 + up(H * D), 8 + 2 * up(H * D)
        self.proj = torch.randn(n, self.v_off + up(H * V), generator=g)
        self.x = torch.randn(n, width, generator=g)
        self.w_gate = torch.randn(2 * H, width, generator=g) * (2.0 / math.sqrt(width))
        self.bias_i, self.bias_f = -1.0 + torch.randn(H, generator=g), 3.0 + 2.0 * torch.randn(H, generator=g)
        if zi is not None:       # the same logits for every token and head, through the biases alone
            self.w_gate.zero_()
            self.bias_i, self.bias_f = torch.full((H,), float(zi)), torch.full((H,), float(zf))
        z = q64(self.x, dt) @ q64(self.w_gate, dt).T
        self.logits = z.float()
        self.i = P.soft_cap(z[:, :H] + self.bias_i.double(), cap)
        self.f = P.log_sigmoid(P.soft_cap(z[:, H:] + self.bias_f.double(), cap))

    def plain(self, a, b, states=None):
        H, D, V = self.H, self.D, self.V
        x = q64(self.proj[a:b], self.dt)
        q = x[:, self.q_off:self.q_off + H * D].reshape(-1, H, D) * D ** -0.5
        k = x[:, self.k_off:self.k_off + H * D].reshape(-1, H, D)
        v = x[:, self.v_off:self.v_off + H * V].reshape(-1, H, V)
        outs = [P.memory_scan(q[:, h], k[:, h], v[:, h], self.i[a:b, h], self.f[a:b, h], None if states is None else states[h]) for h in range(H)]
        return torch.cat([o for o, _ in outs], dim=1), [s for _, s in outs]

    def fresh(self, slots):
        return torch.zeros(slots, self.H, self.D, self.V, device=DEV), torch.zeros(slots, self.H, self.D + 2, device=DEV)

    def run(self, kind, parts, state, tails, columns=0):
        """``parts``: (slot, first row, rows) per sequence, in one launch."""
        o = ops()
        rows = torch.cat([torch.arange(a, a + t) for _, a, t in parts])
        cu = [0]
        for _, _, t in parts:
            cu.append(cu[-1] + t)
        out = torch.full((len(rows), self.H * self.V), float("nan"), device=DEV)
        proj = self.proj[rows].to(self.dt).to(DEV)
        args = (self.bias_i.to(DEV), self.bias_f.to(DEV), self.cap, self.D ** -0.5, out, state, tails, i32(cu), i32([s for s, _, _ in parts]),
                len(parts), self.H, self.D, self.V)
        offs = (self.q_off, self.k_off, self.v_off)
        if kind == "step":
            assert o.mlstm_step(proj, *offs, self.x[rows].to(self.dt).to(DEV), self.w_gate.to(self.dt).to(DEV), *args)
        elif kind == "chunks":
            from builderforce_inference_b200.kernels import fast_ops
            assert fast_ops.mlstm_chunks_bf16(proj, *offs, self.logits[rows].to(DEV), *args, columns=columns)
        else:
            o.mlstm_scan(proj, *offs, self.logits[rows].to(DEV), *args)
        return out.double().cpu()

    def same_state(self, state, tails, slot, plain, tol):
        assert rel_err(state[slot], torch.stack([s for s, _, _ in plain])) < tol
        assert rel_err(tails[slot, :, :self.D], torch.stack([n for _, n, _ in plain])) < tol
        assert rel_err(tails[slot, :, self.D], torch.stack([m for _, _, m in plain])) < tol
        assert int(tails[slot, :, self.D + 1].contiguous().view(torch.int32).abs().max()) == 0      # the counter is back at zero


def head_errors(got, ref, H):
    """Largest error of any token and head, against the head's largest output over the sequence (where n . q,
    which the output is divided by, is near zero: errors of n . q count double there)."""
    g, r = got.reshape(got.shape[0], H, -1), ref.reshape(ref.shape[0], H, -1)
    assert torch.isfinite(g).all()
    return float(((g - r).abs().amax(dim=(0, 2)) / r.abs().amax(dim=(0, 2)).clamp(min=1e-6)).max())


@pytest.mark.parametrize("kind,dt,sizes", [("scan", F32, (3, 10, 6)), ("scan", BF16, (2, 24, 40)), ("scan", F32, (1, 300, 70)), ("scan", F32, (2, 1, 1)),
                                           ("scan", F32, (2, 64, 129)), ("chunks", BF16, (2, 64, 64)), ("chunks", BF16, (3, 128, 32)),
                                           ("chunks", BF16, (1, 48, 16)), ("chunks", BF16, (2, 16, 128)), ("chunks", BF16, (1, 256, 96))])
def test_memory_whole_in_portions_and_token_by_token(kind, dt, sizes):
    """Gates, decays, sums and state are float32 (in effect) in every kernel: only rounded inputs enter."""
    H, D, V = sizes
    n = 203
    mem = Memory(H, D, V, n, dt)
    ref, S_ref = mem.plain(0, n)
    one = "step" if D <= 256 else "scan"
    for cuts in ([n], [64, 1, 2, n - 67], [128, 65, n - 193], [1] * n):
        state, tails = mem.fresh(3)
        state[0].fill_(float("nan"))                      # another slot's state must not matter
        outs, at = [], 0
        for c in cuts:
            outs.append(mem.run(kind if c > 1 else one, [(1, at, c)], state, tails))
            at += c
        assert head_errors(torch.cat(outs), ref, H) < 2e-4, cuts
        mem.same_state(state, tails, 1, S_ref, 2e-5)
        assert float(state[2].abs().max()) == 0.0 and float(tails[2].abs().max()) == 0.0


@pytest.mark.parametrize("columns", [16, 32, 64])
@pytest.mark.parametrize("D", [16, 64, 80, 128])
def test_memory_chunks_with_every_share_of_columns(columns, D):
    mem = Memory(2, D, 64, 150, BF16, seed=columns)
    ref, S_ref = mem.plain(0, 150)
    state, tails = mem.fresh(1)
    got = torch.cat([mem.run("chunks", [(0, a, t)], state, tails, columns) for a, t in ((0, 70), (70, 80))])
    assert head_errors(got, ref, 2) < 2e-4
    mem.same_state(state, tails, 0, S_ref, 2e-5)


@pytest.mark.parametrize("kind,dt,sizes", [("scan", F32, (2, 20, 33)), ("scan", BF16, (2, 32, 48)), ("chunks", BF16, (2, 32, 48)),
                                           ("step", F32, (3, 9, 70)), ("step", BF16, (2, 128, 128)), ("step", BF16, (1, 256, 32))])
def test_memory_in_a_mixed_batch_of_continuations(kind, dt, sizes):
    """Unequal portions of sequences that have a past, in slots out of order, and a padding row without a slot."""
    mem = Memory(*sizes, 420, dt, seed=1)
    past = {4: (0, 0), 0: (128, 37), 2: (165, 60), 1: (226, 64), 3: (300, 5)}          # slot: first row, rows already seen
    new = {4: 128, 0: 24, 2: 1, 1: 10, 3: 115} if kind != "step" else {s: 1 for s in past}
    state, tails = mem.fresh(6)
    parts, refs = [], []
    for slot, (a, t) in past.items():
        before = mem.plain(a, a + t)[1] if t else None
        if t:
            mem.run("scan", [(slot, a, t)], state, tails)
        parts.append((slot, a + t, new[slot]))
        refs.append(mem.plain(a + t, a + t + new[slot], before))
    parts.insert(2, (-1, 0, 1 if kind == "step" else 3))
    got, at = mem.run(kind, parts, state, tails), 0
    for slot, _, t in parts:
        if slot >= 0:
            o, S_end = refs.pop(0)
            assert head_errors(got[at:at + t], o, sizes[0]) < 2e-4, slot
            mem.same_state(state, tails, slot, S_end, 2e-5)
        at += t
    assert float(state[5].abs().max()) == 0.0


@pytest.mark.parametrize("kind,dt", [("scan", F32), ("chunks", BF16), ("step", BF16)])
@pytest.mark.parametrize("zi,zf", [(50.0, 50.0), (-50.0, 50.0), (50.0, -50.0), (-50.0, -50.0), (0.0, 0.0), (-3.0, 8.0)])
def test_memory_at_the_ends_of_its_gates(kind, dt, zi, zf):
    """Gates pressed against their caps: a memory that keeps everything, forgets at once, takes in e^cap or
    e^-cap of its input; the running maximum starts at 0, which a first input gate below it does not move."""
    n = 150
    mem = Memory(2, 16, 32, n, dt, cap=15.0, seed=2, zi=zi, zf=zf)
    ref, S_ref = mem.plain(0, n)
    state, tails = mem.fresh(1)
    if kind == "step":
        got = torch.cat([mem.run("step", [(0, t, 1)], state, tails) for t in range(n)])
    else:
        got = torch.cat([mem.run(kind, [(0, a, t)], state, tails) for a, t in ((0, 65), (65, 2), (67, n - 67))])
    rows = (got - ref).abs().amax(dim=1) / ref.abs().amax(dim=1).clamp(min=1e-9)
    assert torch.isfinite(got).all() and float(rows.max()) < 2e-3
    assert float(rows.median()) < 2e-5
    mem.same_state(state, tails, 0, S_ref, 3e-5)


@pytest.mark.parametrize("kind,dt", [("scan", F32), ("scan", BF16), ("chunks", BF16)])
def test_memory_answers_one_loud_key_far_away(kind, dt):
    """One key and value among silent ones: every later output is that value times k . q over the floor or
    their own product, decayed by the forget gates in between; earlier outputs and the other head stay
    silent.  600 tokens on the answer is still there, over portions and single tokens."""
    H, D, V, n, loud = 2, 32, 16, 600, 70
    mem = Memory(H, D, V, n, dt, cap=30.0, zi=2.0, zf=7.0)
    mem.proj.zero_()
    mem.proj[:, mem.q_off:mem.q_off + D] = 1.0
    mem.proj[loud, mem.k_off:mem.k_off + D] = 0.25
    mem.proj[loud, mem.v_off:mem.v_off + V] = 3.0
    i, f = float(mem.i[0, 0]), float(mem.f[0, 0])
    for cuts in ([n], [60, 5, 300, 235], [loud + 1] + [1] * 9 + [n - loud - 10]):
        state, tails = mem.fresh(1)
        outs, at = [], 0
        for c in cuts:
            outs.append(mem.run(kind if c > 1 else "step", [(0, at, c)], state, tails))
            at += c
        got = torch.cat(outs)
        assert float(got[:loud].abs().max()) == 0.0 and float(got[:, V:].abs().max()) == 0.0
        for t in (loud, loud + 1, loud + 57, loud + 58, 127, 128, n - 1):
            kq = 0.25 * D * D ** -0.5 * math.exp(i + (t - loud) * f)                # in units of 1
            want = 3.0 * kq / max(kq, 1.0)
            assert abs(float(got[t, 0]) - want) < 2e-4, (cuts, t)


@pytest.mark.parametrize("dt", [F32, BF16])
def test_norm_per_head_with_weight_and_a_sigmoid_gate(dt):
    o = ops()
    g = torch.Generator().manual_seed(8)
    for n, H, V in ((5, 3, 7), (9, 1, 64), (2, 16, 128)):
        x = torch.randn(n, H * V, generator=g) * torch.logspace(-4, 1, n)[:, None]       # down to where eps matters
        gate, w = 2.0 * torch.randn(n, H * V + 5, generator=g), 1.0 + 0.3 * torch.randn(H * V, generator=g)
        y = torch.empty(n, H * V, dtype=dt, device=DEV)
        o.gated_group_norm(x.to(DEV), gate.to(dt).to(DEV)[:, 2:2 + H * V], w.to(dt).to(DEV), 1e-5, y, H, gate_first=False,
                           gate_act=o.GATE_SIGMOID)
        ref = P.rms(x.double().view(n, H, V), 1e-5).reshape(n, H * V) * q64(w, dt) * torch.sigmoid(q64(gate, dt)[:, 2:2 + H * V])
        assert rel_err(y, ref) < (1e-6 if dt == F32 else 8e-3)


# ------------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_whole_prompts_and_every_layer_run(name, dtype):
    from builderforce_inference_b200.engine.context import build_context
    eng, cfg, w = engine(name, dtype)
    ids = prompts(cfg["vocab"], [330])[0]
    ref, layers = P.forward(cfg, w, ids, True)
    slot = eng.acquire()
    assert close(eng.step([S(slot, ids)]), ref, dtype)
    eng.release(slot)
    # the sum of the copies after every layer run (a looped layer counts each time)
    slot = eng.acquire()
    eng.cache.begin_step([slot], [len(ids)])
    ctx = build_context([(slot, 0, ids)], eng.dtype, eng.workspace, eng.device, eng.status)
    x = eng.decoder.embed(ctx)
    for i in range(len(P.schedule(cfg))):
        eng.decoder.run_layers(ctx, x, eng.cache, i, i + 1)
        assert close(x.view(len(ids), cfg["streams"], cfg["width"]).sum(dim=1), layers[i], dtype), i
    eng.cache.end_step([slot], [len(ids)])
    eng.release(slot)
    eng.cache.check()
    eng.check_status()


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_prompt_then_token_by_token(name, dtype, graphs):
    eng, cfg, w = engine(name, dtype, use_graphs=graphs)
    ids = prompts(cfg["vocab"], [330], 40)[0]
    ref = P.forward(cfg, w, ids)
    slot = eng.acquire()
    head = 3
    outs = [eng.step([S(slot, ids[:head])]).clone()]
    for t in ids[head:]:
        outs.append(eng.step([S(slot, [t])]).clone())
    assert close(torch.cat(outs), ref, dtype)
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


def test_a_long_prompt_and_long_decoding_in_float32():
    """1,500 tokens, the last 200 one by one."""
    eng, cfg, w = engine("odd", "float32")
    ids = prompts(cfg["vocab"], [1500], 77)[0]
    ref = P.forward(cfg, w, ids)
    slot = eng.acquire()
    outs = [eng.step([S(slot, ids[:1300])]).clone()] + [eng.step([S(slot, [t])]).clone() for t in ids[1300:]]
    assert rel_err(torch.cat(outs), ref) < 5e-5


def plain_in_float32(cfg, w, ids):
    wide, P.F = P.F, F32
    try:
        return P.forward(cfg, w, ids)
    finally:
        P.F = wide


@pytest.mark.parametrize("seed", range(501, 525))
def test_random_configurations_in_float32(seed):
    """Configurations drawn from a seed (layer order, every size, copies, loops, caps, rotation, with and
    without feed-forward): an unequal batch of prompts, five tokens decoded together, and the longest
    prompt again in portions, against the plain implementation.  Some draws amplify rounding (a memory divides
    by n . q, which may be near zero), so the bound is ten times the plain implementation's own error in
    float32 where that is more than 4e-4."""
    from builderforce_inference_b200.engine.engine import Engine
    cfg = random_config(seed)
    w = make_weights(cfg, seed, F32)
    eng = Engine.load(write_folder(cfg, w), dtype="float32", max_tokens=2048)
    w64 = {k: v.to(torch.float64) for k, v in w.items()}
    lens = [(1, 5, 70, 130, 260)[seed % 5], (2, 33, 200)[seed % 3], (1, 64, 129)[seed % 2]]
    seqs = prompts(cfg["vocab"], [n + 5 for n in lens], seed)
    refs = [P.forward(cfg, w64, s) for s in seqs]
    tol = max([4e-4] + [10.0 * rel_err(plain_in_float32(cfg, w, s), r) for s, r in zip(seqs, refs)])
    assert tol < 1e-2
    slots = [eng.acquire() for _ in seqs]
    got = eng.step([S(sl, s[:n]) for sl, s, n in zip(slots, seqs, lens)])
    assert rel_err(got, torch.cat([r[:n] for r, n in zip(refs, lens)])) < tol, cfg
    for step in range(5):
        got = eng.step([S(sl, [s[n + step]]) for sl, s, n in zip(slots, seqs, lens)])
        assert rel_err(got, torch.stack([r[n + step] for r, n in zip(refs, lens)])) < tol, (step, cfg)
    for sl in slots:
        eng.release(sl)
    i = max(range(3), key=lambda k: lens[k])
    sl, outs, at = eng.acquire(), [], 0
    for c in [max(1, lens[i] // 3), 2, 1, 97, 10 ** 6]:
        c = min(c, lens[i] - at)
        if c > 0:
            outs.append(eng.step([S(sl, seqs[i][at:at + c])]).clone())
            at += c
    assert rel_err(torch.cat(outs), refs[i][:lens[i]]) < tol, cfg
    eng.release(sl)
    eng.cache.check()
    eng.check_status()


@pytest.mark.parametrize("seed", range(601, 613))
def test_random_configurations_in_bfloat16(seed):
    """The same draw in bfloat16: a prompt whole, in portions and its end token by token stay close to the
    plain implementation."""
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
    from zitezen_models import ZT_ODD
    eng = Engine.from_random(ZT_ODD, 5, dtype="bfloat16", cache_bytes=1 << 24, cache_slots=4)
    memories = {0: (3, 9, 5), 1: (2, 7, 20), 3: (5, 24, 6), 4: (1, 20, 36)}
    held = sum(4 * H * (D * V + D + 2) for i in P.schedule(ZT_ODD) if i in memories for H, D, V in [memories[i]])
    assert eng.cache_plan.n_slots == 4 and eng.cache_plan.state_bytes_per_slot == held
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

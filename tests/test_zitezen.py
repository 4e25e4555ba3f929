"""Zitezen without a GPU: the configuration reader and its refusals by key, the model as data, what its
blocks ask of the cache, what the parts refuse, and the plain implementation
(tests/plain/zitezen_plain.py) against closed forms."""
import copy
import math

import pytest
import torch

from plain import zitezen_plain as P
from zitezen_models import ZT_ODD, ZT_WIDE, make_weights, prompts, random_config, tensor_shapes

from builderforce_inference_b200.cache import SequenceCache
from builderforce_inference_b200.cache.pages import CacheError
from builderforce_inference_b200.config.base import ConfigError
from builderforce_inference_b200.config.zitezen import ZitezenConfig, ZitezenLatent, ZitezenMemory, ZitezenParallel
from builderforce_inference_b200.engine.decoder import Decoder, Runtime, expected_tensors
from builderforce_inference_b200.parts.base import BLOCKS, MIXERS, KVNeed, PartSpec, StateNeed
from builderforce_inference_b200.registry import architecture_for, describe_model

F = torch.float64


# ------------------------------------------------------------------------------------------------ configuration
def test_config_reads_every_size_and_constant():
    c = ZitezenConfig.from_dict(ZT_ODD)
    assert (c.vocab, c.width, c.streams, c.eps, len(c.layers), c.loop) == (137, 42, 3, 3e-5, 6, (1, 4, 2))
    assert c.order == (0, 1, 2, 3, 1, 2, 3, 4, 5)
    p = c.layers[0].mixer
    assert isinstance(p, ZitezenParallel) and (p.left_scale, p.right_scale) == (0.7, 1.4)
    a = p.left
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.rot.base, a.rot.dims) == (6, 2, 10, 14, 0.35, 3.0, 90.0, 6)
    assert p.right == ZitezenMemory(heads=3, dim=9, vdim=5, gate_cap=6.0)
    assert c.layers[1].mixer == ZitezenMemory(heads=2, dim=7, vdim=20, gate_cap=4.0) and c.layers[1].ff == 26
    m = c.layers[2].mixer
    assert isinstance(m, ZitezenLatent) and c.layers[2].ff is None
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank, m.scale, m.rot.base, m.rot.dims) == (3, 10, 6, 14, 22, 18, 0.24, 700.0, 6)
    assert c.layers[4].mixer.left.rot is None
    assert architecture_for(ZT_ODD).name == "zitezen"
    bare = copy.deepcopy(ZT_ODD)
    del bare["loop"], bare["layers"][0]["mixer"]["left"]["softcap"]
    c = ZitezenConfig.from_dict(bare)
    assert c.order == tuple(range(6)) and c.layers[0].mixer.left.softcap is None


def _changed(path, value):
    cfg = copy.deepcopy(ZT_ODD)
    node = cfg
    for k in path[:-1]:
        node = node[k]
    if value is KeyError:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path,value,names", [
    (("vocab",), KeyError, "vocab"),
    (("streams",), 0, "streams"),
    (("streams",), 33, "streams"),
    (("norm",), KeyError, "norm"),
    (("norm", "eps"), 0.0, "eps"),
    (("layers",), [], "layers"),
    (("loop", "stop"), 7, "6 layers"),
    (("loop", "start"), 5, "6 layers"),
    (("loop", "times"), 0, "times"),
    (("layers", 0, "type"), "attention", "type"),
    (("layers", 0, "mixer", "left", "kv_heads"), 4, "kv_heads"),
    (("layers", 0, "mixer", "left", "dim"), 9, "dim"),
    (("layers", 0, "mixer", "left", "softcap"), 0.0, "softcap"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 12, "dims"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 5, "dims"),
    (("layers", 0, "mixer", "right"), KeyError, "right"),
    (("layers", 0, "mixer", "right", "gate_cap"), -1.0, "gate_cap"),
    (("layers", 1, "mixer", "gate_cap"), KeyError, "gate_cap"),
    (("layers", 1, "mixer", "heads"), 0, "heads"),
    (("layers", 2, "mixer", "q_rank"), KeyError, "q_rank"),
    (("layers", 2, "mixer", "kv_rank"), 23, "kv_rank"),
    (("layers", 2, "mixer", "rot", "dims"), 8, "dims"),
    (("layers", 1, "mlp", "kind"), "moe", "kind"),
    (("layers", 1, "mlp", "ff"), 0, "ff"),
])
def test_config_refuses_by_key(path, value, names):
    with pytest.raises(ConfigError) as e:
        ZitezenConfig.from_dict(_changed(path, value))
    assert names in str(e.value)


# ------------------------------------------------------------------------------------------------ the model as data
@pytest.mark.parametrize("cfg", [ZT_ODD, ZT_WIDE] + [random_config(s) for s in range(500, 525)])
def test_spec_names_every_tensor_with_its_shape(cfg):
    spec = describe_model(cfg)
    want, have = expected_tensors(spec), tensor_shapes(cfg)
    assert set(want) == set(have)
    for name, (shape, _) in have.items():
        assert tuple(want[name].shape) == tuple(shape), name
    assert spec.head_name == "head" and spec.streams == cfg["streams"]
    assert [r.layer for r in spec.schedule] == P.schedule(cfg) and all(r.cache_of is None for r in spec.schedule)
    for i, lay in enumerate(cfg["layers"]):       # what surrounds a feed-forward the layer does not have may be in the file all the same
        assert (f"l{i}.norm2.alpha" in spec.ignored_names) == (f"l{i}.hc2.mix" in spec.ignored_names) == (lay["mlp"] is None)
    assert Decoder(spec, Runtime(torch.device("cpu"), torch.float32)).graph_safe()


def test_every_pass_of_a_loop_has_a_state_of_its_own():
    spec = describe_model(ZT_ODD)
    needs = [BLOCKS.build(layer.block).cache_need() for layer in spec.layers]
    assert needs[0] == (KVNeed(2, 10, v_dim=14), StateNeed((3, 9, 5), "float32"), StateNeed((3, 11), "float32"))
    assert needs[1] == (StateNeed((2, 7, 20), "float32"), StateNeed((2, 9), "float32"))
    assert needs[2] == KVNeed(1, 28, v_dim=22, values_in_keys=True)
    d = Decoder(spec, Runtime(torch.device("cpu"), torch.float32))
    c = SequenceCache(d.run_needs(), d.run_cache_of(), 512, 512, torch.float32, torch.device("cpu"))
    first, second = c.run_cache(1), c.run_cache(4)        # the same layer, two passes
    assert [tuple(e.shape[1:]) for e in first.entries] == [(2, 7, 20), (2, 9)]
    assert all(a.data_ptr() != b.data_ptr() for a, b in zip(first.entries, second.entries))
    assert c.run_cache(2).kv.k.data_ptr() != c.run_cache(5).kv.k.data_ptr()
    s = c.acquire()
    for e in first.entries:
        e[s].fill_(3.0)
    c.begin_step([s], [70])
    c.end_step([s], [70])
    with pytest.raises(CacheError, match="fixed size"):
        c.rewind(s, 10)
    c.release(s)
    assert c.acquire() == s and all(float(e[s].abs().max()) == 0.0 for e in first.entries)      # a taken slot starts from zero


def test_parts_refuse_combinations_no_kernel_has():
    with pytest.raises(ValueError, match="cap"):
        MIXERS.build(PartSpec("mlstm", {"width": 8, "n_heads": 1, "dim": 8, "vdim": 8, "gate_cap": 0.0}))
    with pytest.raises(ValueError, match="cap"):
        MIXERS.build(PartSpec("attention", {"width": 8, "n_heads": 1, "n_kv_heads": 1, "head_dim": 8, "softcap": -2.0}))
    norm = PartSpec("dynamic_tanh", {"width": 8})
    mix = PartSpec("mlstm", {"width": 8, "n_heads": 1, "dim": 8, "vdim": 8, "gate_cap": 5.0})
    with pytest.raises(ValueError, match="norm"):
        BLOCKS.build(PartSpec("hyper", {"width": 8, "streams": 2, "norm1": norm, "mixer": mix, "norm2": norm}))
    with pytest.raises(ValueError, match="times"):
        BLOCKS.build(PartSpec("hyper", {"width": 8, "streams": 40, "norm1": norm, "mixer": mix}))


# ------------------------------------------------------------------------------------------------ the plain implementation
def test_plain_memory_against_its_closed_form():
    """Without the running maximum: S and n are sums of ``e^(i_j + f_(j+1) + .. + f_t) k_j (v_j)``, the denominator
    is ``max(|n . q|, 1)`` and the small constant counts in units of ``e^m``."""
    g = torch.Generator().manual_seed(4)
    T, d, dv = 40, 5, 7
    q, k, v = (torch.randn(T, n, generator=g, dtype=F) for n in (d, d, dv))
    i, f = 2.0 * torch.randn(T, generator=g, dtype=F), P.log_sigmoid(2.0 + 2.0 * torch.randn(T, generator=g, dtype=F))
    o, (S, n, m) = P.memory_scan(q, k, v, i, f)
    for t in (0, 1, 17, 39):
        weight = torch.exp(i[:t + 1] + f[:t + 1].sum() - torch.cumsum(f[:t + 1], 0))
        num = (weight[:, None] * (k[:t + 1] @ q[t])[:, None] * v[:t + 1]).sum(0)
        den = (weight * (k[:t + 1] @ q[t])).sum()
        m_t = max([float(f[:t + 1].sum())] + [float(i[j] + f[j + 1:t + 1].sum()) for j in range(t + 1)])
        want = num / (torch.maximum(den.abs(), torch.ones((), dtype=F)) + 1e-6 * math.exp(m_t))
        assert torch.allclose(o[t], want, atol=1e-12)
    assert torch.isclose(m, torch.tensor(m_t, dtype=F))
    # in two pieces, the state handed over
    a, state = P.memory_scan(q[:13], k[:13], v[:13], i[:13], f[:13])
    b, (S2, n2, m2) = P.memory_scan(q[13:], k[13:], v[13:], i[13:], f[13:], state)
    assert torch.equal(torch.cat([a, b]), o) and torch.equal(S, S2) and torch.equal(n, n2) and torch.equal(m, m2)


def test_plain_caps_gates_and_rotations():
    z = torch.tensor([-1e3, -3.0, 0.0, 2.0, 1e3], dtype=F)
    assert torch.allclose(P.soft_cap(z, 5.0), torch.tensor([-5.0, -5 * math.tanh(0.6), 0.0, 5 * math.tanh(0.4), 5.0], dtype=F))
    assert torch.allclose(P.log_sigmoid(z)[1:4], torch.log(1 / (1 + torch.exp(-z[1:4])))) and float(P.log_sigmoid(z)[0]) == -1e3
    w = {"i": torch.tensor([[30.0]], dtype=F), "i.b": torch.tensor([0.5], dtype=F), "f": torch.tensor([[-30.0]], dtype=F),
         "f.b": torch.tensor([0.0], dtype=F)}
    i, f = P.memory_gates(w, "", {"gate_cap": 4.0}, torch.ones(1, 1, dtype=F))
    assert abs(float(i) - 4.0) < 1e-5 and abs(float(f) + math.log1p(math.exp(4.0))) < 1e-5
    g = torch.Generator().manual_seed(1)
    x, y = (torch.randn(2, 1, 6, generator=g, dtype=F) for _ in range(2))
    for turn in (P.rotate_halves, P.rotate_neighbours):      # a score depends on the distance only, and the rest of a head stays
        def score(p, q):
            a, b = (turn(v[:1], *P.rotary_angles([n], 4, 50.0), 4) for v, n in ((x, p), (y, q)))
            return float((a[0, 0] * b[0, 0]).sum())
        assert abs(score(9, 2) - score(507, 500)) < 1e-9 and abs(score(9, 2) - score(9, 3)) > 1e-6
        assert torch.equal(turn(x, *P.rotary_angles([3, 4], 4, 50.0), 4)[..., 4:], x[..., 4:])
    assert torch.equal(P.rotate_halves(x, *P.rotary_angles([3, 4], 2, 50.0), 2), P.rotate_neighbours(x, *P.rotary_angles([3, 4], 2, 50.0), 2))


def test_plain_copies_with_the_identity_are_an_ordinary_residual_stream():
    """Copies that keep to themselves, read as their mean and written alike, stay equal: the stream then is the
    ordinary one times the number of copies."""
    g = torch.Generator().manual_seed(2)
    x, y = (torch.randn(4, 6, generator=g, dtype=F) for _ in range(2))
    one = torch.ones(3, dtype=F)
    X = P.connect(x[None].repeat(3, 1, 1), one / 3, one, torch.eye(3, dtype=F), lambda u: torch.sin(u) + y)
    assert torch.allclose(X, (x + torch.sin(x) + y)[None].repeat(3, 1, 1))
    # the matrix is indexed [from, to]
    mix = torch.zeros(2, 2, dtype=F)
    mix[0, 1] = 1.0
    X = P.connect(torch.stack([x, y]), torch.tensor([0.0, 1.0], dtype=F), torch.tensor([2.0, 0.0], dtype=F), mix, lambda u: u)
    assert torch.equal(X[0], 2.0 * y) and torch.equal(X[1], x)


def test_plain_model_is_causal_and_loops():
    cfg = copy.deepcopy(ZT_ODD)
    w = {k: v.to(F) for k, v in make_weights(cfg, 2, torch.float32).items()}
    ids = prompts(cfg["vocab"], [30])[0]
    full, layers = P.forward(cfg, w, ids, True)
    assert torch.allclose(P.forward(cfg, w, ids[:17]), full[:17]) and layers.shape == (9, 30, 42)
    cfg["loop"] = None
    assert float((P.forward(cfg, w, ids) - full).abs().max()) > 1e-2
    cfg["loop"] = {"start": 2, "stop": 2, "times": 3}
    assert torch.equal(P.forward(cfg, w, ids), P.forward(dict(cfg, loop=None), w, ids))

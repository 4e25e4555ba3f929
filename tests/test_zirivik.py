"""Zirivik without a GPU: the configuration reader and its refusals by key, the model as data, what its
blocks ask of the cache, what the cache keeps for readers with other masks, and the plain
implementation (tests/plain/zirivik_plain.py) against closed forms."""
import copy
import math
import random

import pytest
import torch

from plain import zirivik_plain as P
from zirivik_models import ZV_ODD, ZV_WIDE, make_weights, random_config, tensor_shapes

from builderforce_inference_b200.cache import SequenceCache
from builderforce_inference_b200.cache.pages import CacheError, PageTable
from builderforce_inference_b200.config.base import ConfigError
from builderforce_inference_b200.config.zirivik import (ZirivikAttention, ZirivikConfig, ZirivikDense, ZirivikMoE,
                                                         ZirivikRetention)
from builderforce_inference_b200.engine.decoder import expected_tensors
from builderforce_inference_b200.kernels.ops import KernelError
from builderforce_inference_b200.parts.base import BLOCKS, FEED_FORWARDS, MIXERS, KVNeed, PartSpec, StateNeed
from builderforce_inference_b200.registry import architecture_for, describe_model

F = torch.float64


# ------------------------------------------------------------------------------------------------ configuration
def test_config_reads_every_size_and_constant():
    c = ZirivikConfig.from_dict(ZV_ODD)
    assert (c.vocab, c.width, c.eps, c.embedding_scale, c.logit_softcap, len(c.layers)) == (131, 40, 2e-5, 3.3, 7.0, 6)
    a = c.layers[0].mixer
    assert isinstance(a, ZirivikAttention)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.keep_first, a.kv_from) == (4, 2, 24, 10, 0.21, 9, 3, None)
    assert c.layers[2].mixer.kv_from == 0 and c.layers[2].mixer.keep_first == 130 and c.layers[2].mlp is None
    r = c.layers[1].mixer
    assert isinstance(r, ZirivikRetention)
    assert (r.heads, r.dim, r.vdim, r.decay, r.rot_base, r.rot_dims) == (3, 10, 6, (0.5, 0.9, 0.999), 100.0, 6)
    assert c.layers[1].mlp == ZirivikDense(ff=36) and c.layers[3].mlp == ZirivikMoE(experts=7, top=1, ff=12, limit=2.5)
    assert architecture_for(ZV_ODD).name == "zirivik"
    bare = copy.deepcopy(ZV_ODD)
    del bare["embedding"], bare["logit_softcap"], bare["layers"][4]["mixer"]["mask"], bare["layers"][1]["mixer"]["rot"]
    c = ZirivikConfig.from_dict(bare)
    assert c.embedding_scale == 1.0 and c.logit_softcap is None and c.layers[4].mixer.window is None and c.layers[1].mixer.rot_base is None
    assert describe_model(bare).logit_softcap is None


def _changed(path, value):
    cfg = copy.deepcopy(ZV_ODD)
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
    (("norm",), KeyError, "norm"),
    (("layers",), [], "layers"),
    (("logit_softcap",), 0.0, "logit_softcap"),
    (("layers", 0, "type"), "mamba", "type"),
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "dim"), 9, "dim"),
    (("layers", 0, "mixer", "mask", "size"), 0, "size"),
    (("layers", 0, "mixer", "mask", "keep_first"), -1, "keep_first"),
    (("layers", 1, "mixer", "decay"), [0.5, 0.9], "decay"),
    (("layers", 1, "mixer", "decay"), [0.5, 0.9, 1.5], "decay"),
    (("layers", 1, "mixer", "rot", "dims"), 12, "dims"),
    (("layers", 1, "mixer", "rot", "dims"), 5, "dims"),
    (("layers", 2, "mixer", "kv_from"), 1, "kv_from"),         # a retention layer has no keys to lend
    (("layers", 2, "mixer", "kv_from"), 4, "kv_from"),         # a later layer
    (("layers", 5, "mixer", "kv_from"), 2, "kv_from"),         # a layer that borrows itself
    (("layers", 5, "mixer", "kv_from"), 0, "kv_from"),         # other head counts
    (("layers", 0, "mlp", "kind"), "glu", "kind"),
    (("layers", 0, "mlp", "router", "top"), 6, "top"),
    (("layers", 0, "mlp", "expert"), KeyError, "expert"),
    (("layers", 0, "mlp", "expert", "limit"), 0.0, "limit"),
    (("layers", 1, "mlp", "ff"), 0, "ff"),
])
def test_config_refuses_by_key(path, value, names):
    with pytest.raises(ConfigError) as e:
        ZirivikConfig.from_dict(_changed(path, value))
    assert names in str(e.value)


# ------------------------------------------------------------------------------------------------ the model as data
@pytest.mark.parametrize("cfg", [ZV_ODD, ZV_WIDE] + [random_config(s) for s in range(300, 320)])
def test_spec_names_every_tensor_with_its_shape(cfg):
    spec = describe_model(cfg)
    want = expected_tensors(spec)
    have = tensor_shapes(cfg)
    assert set(want) == set(have)
    for name, (shape, _) in have.items():
        assert tuple(want[name].shape) == tuple(shape), name
    assert spec.head_name is None and spec.embedding_scale == cfg["embedding"]["scale"]
    assert [r.cache_of for r in spec.schedule] == [lay["mixer"].get("kv_from") for lay in cfg["layers"]]
    # the norms of a feed-forward a layer does not have may be in the file all the same
    for i, lay in enumerate(cfg["layers"]):
        assert (f"l{i}.norm2" in spec.ignored_names) == (lay["mlp"] is None)


def test_blocks_ask_for_their_masks_and_states():
    spec = describe_model(ZV_ODD)
    needs = [BLOCKS.build(layer.block).cache_need() for layer in spec.layers]
    assert needs[0] == KVNeed(2, 24, 9, v_dim=10, keep_first=3)
    assert needs[1] == StateNeed((3, 10, 6), "float32")
    assert needs[2] == KVNeed(2, 24, 70, v_dim=10, keep_first=130)
    assert needs[4] == KVNeed(3, 16, 64, v_dim=28)


def test_parts_refuse_combinations_no_kernel_has():
    with pytest.raises(ValueError, match="chunk"):
        MIXERS.build(PartSpec("attention", {"width": 8, "n_heads": 1, "n_kv_heads": 1, "head_dim": 8, "chunk": 4, "keep_first": 2}))
    with pytest.raises(ValueError, match="gate"):
        MIXERS.build(PartSpec("lightning", {"width": 8, "n_heads": 1, "dim": 8, "vdim": 8, "decay": [0.5], "gate": "silu"}))
    with pytest.raises(ValueError, match="halves"):
        MIXERS.build(PartSpec("lightning", {"width": 8, "n_heads": 1, "dim": 8, "vdim": 8, "decay": [0.5],
                                            "position": PartSpec("rotary", {"theta": 10.0, "rot_dim": 8, "pairing": "adjacent"})}))
    with pytest.raises(ValueError, match="bias"):
        FEED_FORWARDS.build(PartSpec("dense_mlp", {"width": 8, "inner": 8, "activation": "relu_squared"}))
    with pytest.raises(ValueError, match="input"):
        FEED_FORWARDS.build(PartSpec("mixture_of_experts", {"width": 8, "n_experts": 2, "top": 1, "inner": 4, "shared_inner": 4,
                                                            "weight_on": "input"}))
    with pytest.raises(ValueError, match="clamp"):
        FEED_FORWARDS.build(PartSpec("mixture_of_experts", {"width": 8, "n_experts": 2, "top": 1, "inner": 4, "expert": "relu_squared",
                                                            "limit": 1.0}))
    from builderforce_inference_b200.kernels import linear
    with pytest.raises(KernelError, match="input factors"):
        linear.linear(torch.zeros(2, 4), torch.zeros(6, 4), torch.zeros(2, 6), linear.EPI_STORE, in_scale=(torch.ones(2, 1), 6))


# ------------------------------------------------------------------------------------------------ what the cache keeps
@pytest.mark.parametrize("window,keep", [(9, 3), (64, 64), (64, 65), (100, 130), (1, 1), (200, 0), (1, 200)])
def test_page_table_keeps_the_first_positions_and_the_window(window, keep):
    t = PageTable(64, window, None, keep)
    t.open(0)
    rng = random.Random(window * 1000 + keep)
    n = 0
    while n < 700:
        step = rng.choice([1, 1, 1, 2, 63, 64, 65, 130])
        t.ensure(0, n, n + step)
        # every position that a token of the step reads has its page
        for p in (n, n + step - 1):
            for j in range(p + 1):
                if p - j < window or j < keep:
                    assert t.rows[0][j // 64] >= 0, (p, j)
        n += step
        t.trim(0, n)
        held = {b for b, page in enumerate(t.rows[0]) if page >= 0}
        want = {j // 64 for j in range(n) if n - j < window or j < keep}
        assert held >= want
        assert held <= want | set(range((keep + 63) // 64)) | {(n - 1) // 64, n // 64}
        assert t.kept_positions(n) == sum(1 for j in range(n) if n - j < window or j < keep)
        t.check()
    t.close(0)
    assert t.pool.n_free == 64


def _cache(needs, cache_of, **kw):
    return SequenceCache(needs, cache_of, kw.pop("max_tokens", 2048), kw.pop("max_seq_len", 2048), torch.float32, torch.device("cpu"), **kw)


def test_a_borrowing_run_reads_under_its_own_mask_and_the_lender_keeps_enough():
    lend, near, far = KVNeed(2, 8, 9, keep_first=3), KVNeed(2, 8, 4, keep_first=1), KVNeed(2, 8, 200, keep_first=70)
    c = _cache([lend, near, far, lend], [None, 0, 0, None])
    views = [c.run_cache(r).kv for r in range(4)]
    assert [(v.window, v.keep_first) for v in views] == [(9, 3), (4, 1), (200, 70), (9, 3)]
    assert views[1].k.data_ptr() == views[0].k.data_ptr() == views[2].k.data_ptr() != views[3].k.data_ptr()
    assert [c.run_cache(r).writes_cache for r in range(4)] == [True, False, False, True]
    s = c.acquire()
    c.begin_step([s], [500])
    c.end_step([s], [500])
    groups = {id(g): g for g in c.kv_groups}
    assert len(groups) == 2
    wide = next(g for g in c.kv_groups if g.runs == [0])
    thin = next(g for g in c.kv_groups if g.runs == [3])
    assert (wide.need.window, wide.need.keep_first) == (200, 70) and (thin.need.window, thin.need.keep_first) == (9, 3)
    assert [b for b, p in enumerate(wide.table.rows[s]) if p >= 0] == [0, 1, 4, 5, 6, 7]
    assert [b for b, p in enumerate(thin.table.rows[s]) if p >= 0] == [0, 7]
    c.release(s)
    c.check()


def test_a_borrower_without_a_window_makes_the_lender_keep_everything():
    c = _cache([KVNeed(1, 8, 5, keep_first=2), KVNeed(1, 8)], [None, 0])
    g = c.kv_groups[0]
    assert g.need.window is None and g.table.keeps_everything
    assert c.run_cache(0).kv.window == 5 and c.run_cache(0).kv.keep_first == 2 and c.run_cache(1).kv.window is None
    with pytest.raises(CacheError, match="cannot read"):
        _cache([KVNeed(1, 8, 5), KVNeed(1, 16, 5)], [None, 0])


# ------------------------------------------------------------------------------------------------ the plain implementation
def test_plain_mask_and_recurrence_against_closed_forms():
    m = P.window_mask(12, 4, 2)
    assert m[11].tolist() == [True, True] + [False] * 6 + [True] * 4 and m[0].tolist() == [True] + [False] * 11
    assert m[5].tolist() == [True] * 6 + [False] * 6            # positions 0, 1 kept; 2..5 in the window
    assert torch.equal(P.window_mask(5), torch.tril(torch.ones(5, 5)).bool())
    # o_t = sum_j decay^(t-j) (q_t . k_j) v_j
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, n, generator=g, dtype=F) for n in (3, 3, 4))
    decay = torch.tensor([0.5, 0.9], dtype=F)
    o, _ = P.decayed_recurrence(q, k, v, decay)
    for h in range(2):
        want = sum(decay[h] ** (8 - j) * (q[8, h] @ k[j, h]) * v[j, h] for j in range(9))
        assert torch.allclose(o[8, h], want)
    # scores depend on the distance only: turning q and k at shifted positions changes nothing
    a = P.rotate_half(q, range(0, 9), 50.0, 2)
    b = P.rotate_half(k, range(0, 9), 50.0, 2)
    a2, b2 = P.rotate_half(q, range(700, 709), 50.0, 2), P.rotate_half(k, range(700, 709), 50.0, 2)
    assert torch.allclose(a[8, 0] @ b[3, 0], a2[8, 0] @ b2[3, 0]) and not torch.allclose(a[8, 0] @ b[3, 0], q[8, 0] @ k[3, 0])


def test_plain_feed_forwards_and_cap():
    w = {"m.router": torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F)}
    for e in range(2):
        w.update({f"m.e{e}.gate": torch.eye(2, dtype=F) * (e + 1), f"m.e{e}.up": torch.eye(2, dtype=F), f"m.e{e}.down": torch.eye(2, dtype=F)})
    h = torch.tensor([[0.5, 3.0]], dtype=F)
    y = P.routed_ff(h, w, "m.", {"router": {"experts": 2, "top": 1}, "expert": {"limit": 1.0}})
    s = 1 / (1 + math.exp(-3.0))
    ref = []
    for x in (0.5, 3.0):                                  # expert 1, input scaled by its score; gate and up clamped at 1
        gate, up = min(2 * x * s, 1.0), max(-1.0, min(1.0, x * s))
        ref.append(gate / (1 + math.exp(-1.702 * gate)) * (up + 1))
    assert torch.allclose(y, torch.tensor([ref], dtype=F))
    assert torch.allclose(P.dense_ff(torch.tensor([[1.0, -2.0]], dtype=F), {"u.up": torch.eye(2, dtype=F), "u.down": torch.eye(2, dtype=F)}, "u."),
                          torch.tensor([[1.0, 0.0]], dtype=F))
    cfg = copy.deepcopy(ZV_ODD)
    w = {k: v.to(F) for k, v in make_weights(cfg, 2, torch.float32).items()}
    capped = P.forward(cfg, w, range(20))
    del cfg["logit_softcap"]
    raw = P.forward(cfg, w, range(20))
    assert float(raw.abs().max()) > 7.0 > float(capped.abs().max()) and torch.allclose(capped, 7.0 * torch.tanh(raw / 7.0))

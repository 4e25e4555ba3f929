"""Shared by the Zirivik tests: small configurations with sizes of their own, weights made here
(larger than the package's random fill, so that softmaxes are sharp and routers decide), and model
folders written from them."""
import json
import math
import os
import struct
import tempfile

import torch

F32, BF16 = torch.float32, torch.bfloat16


def ret(dim, vdim, decay, rot=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "retention", "mixer": m}


def att(heads, kv_heads, dim, vdim, scale, size, keep, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size, "keep_first": keep}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(vocab, width, eps, scale, cap, layers):
    return {"architecture": "Zirivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_softcap": cap, "layers": [dict(lay, mlp=mlp) for lay, mlp in layers]}


# odd sizes everywhere: an attention layer first, lending its keys to a layer that looks further back
# and keeps more first tokens than itself; windows shorter than a page, a page long and longer; kept
# first tokens within a page, over two page borders and none; values wider and narrower than the
# keys; rotation over part of a head; top 1, 3 and all experts; layers without feed-forward
ZV_ODD = config(131, 40, 2e-5, 3.3, 7.0, [
    (att(4, 2, 24, 10, 0.21, 9, 3), moe(5, 3, 20, 0.8)),
    (ret(10, 6, (0.5, 0.9, 0.999), (100.0, 6)), dense(36)),
    (att(4, 2, 24, 10, 0.3, 70, 130, kv_from=0), None),
    (ret(24, 40, (0.97, 0.85), (5000.0, 24)), moe(7, 1, 12, 2.5)),
    (att(3, 3, 16, 28, 0.25, 64, 0), dense(20)),
    (att(3, 3, 16, 28, 0.4, 1, 5, kv_from=4), moe(2, 2, 16, 0.3)),
])
# sizes nearer to a served model's, taken by the tensor-core kernels: heads of 64 and 128, windows that
# cross pages, a borrower with a narrower mask than its lender
ZV_WIDE = config(300, 128, 1e-6, 11.0, 20.0, [
    (ret(64, 64, (0.98, 0.999), (1e4, 64)), moe(8, 2, 64, 1.5)),
    (att(8, 2, 64, 64, 0.125, 100, 70), dense(192)),
    (att(8, 2, 64, 64, 0.2, 30, 4, kv_from=1), moe(6, 3, 48, 0.7)),
    (ret(128, 32, (0.9, 0.96, 0.99, 0.9995), (1e5, 32)), None),
    (att(4, 1, 128, 128, 0.088, 130, 10), dense(160)),
])
CONFIGS = {"odd": ZV_ODD, "wide": ZV_WIDE}


def tensor_shapes(cfg):
    """name -> (shape, kind) of every tensor of a Zirivik model, from its config alone."""
    w = cfg["width"]
    out = {"embed": ((cfg["vocab"], w), "table"), "final.norm": ((w,), "norm0")}
    for i, layer in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", layer["mixer"], f"l{i}.mix."
        for s in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            out[p + s] = ((w,), "norm0")
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        out.update({q + "q": ((H * d, w), "matrix"), q + "o": ((w, H * dv), "matrix")})
        if layer["type"] == "retention":
            out.update({q + "k": ((H * d, w), "matrix"), q + "v": ((H * dv, w), "matrix"), q + "g": ((H * dv, w), "matrix")})
        elif "kv_from" not in m:
            out.update({q + "k": ((m["kv_heads"] * d, w), "matrix"), q + "v": ((m["kv_heads"] * dv, w), "matrix")})
        f = layer["mlp"]
        if f is None:
            continue
        q = p + "mlp."
        if f["kind"] == "dense":
            out.update({q + "up": ((f["ff"], w), "matrix"), q + "down": ((w, f["ff"]), "matrix")})
        else:
            ff = f["expert"]["ff"]
            out[q + "router"] = ((f["router"]["experts"], w), "router")
            for e in range(f["router"]["experts"]):
                out.update({f"{q}e{e}.gate": ((ff, w), "expert"), f"{q}e{e}.up": ((ff, w), "expert"), f"{q}e{e}.down": ((w, ff), "expert")})
    return out


def make_weights(cfg, seed, dt, steady=False):
    """``steady``: experts of a layer that resemble one another and milder matrices, for the bfloat16
    models: rounding may turn a close choice between experts, and must then not turn the output with it."""
    g = torch.Generator().manual_seed(seed)
    out, common = {}, {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if kind == "norm0":
            t = 0.25 * t
        elif kind == "table":
            t = 0.7 * t
        elif kind == "router":
            t = t * (1.5 / math.sqrt(shape[1]))
        else:
            if kind == "expert" and steady:
                key = (name.split(".")[0], name.split(".")[-1])
                base = common.setdefault(key, torch.randn(shape, generator=g))
                t = 0.95 * base + 0.2 * t
            t = t * ((1.0 if steady else 1.6) / math.sqrt(shape[1]))
        out[name] = t.to(dt)
    return out


def write_folder(cfg, weights):
    folder = tempfile.mkdtemp(prefix="bfi_zirivik_")
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, t in weights.items():
        raw = t.contiguous().view(torch.int16 if t.dtype == BF16 else torch.int32).numpy().tobytes()
        header[name] = {"dtype": {F32: "F32", BF16: "BF16"}[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return folder


_MODELS = {}


def model(name, dtype, seed=3):
    """(folder, config, float64 weights as stored) of a test model; the store is the run dtype's."""
    key = (name, dtype, seed)
    if key not in _MODELS:
        cfg = CONFIGS[name]
        w = make_weights(cfg, seed, F32 if dtype == "float32" else BF16, steady=dtype != "float32")
        _MODELS[key] = (write_folder(cfg, w), cfg, {k: v.to(torch.float64) for k, v in w.items()})
    return _MODELS[key]


def prompts(vocab, lengths, seed=5):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lengths]


def random_config(seed):
    """A configuration drawn from a seed: two to six layers of both kinds in any order, sizes from
    lists that hold odd ones and values that make other sizes equal or 1, windows from 1 position to
    more than the prompts, kept first tokens from none to more than the window, borrowed keys under
    other masks, rotation over a whole head, a part of it or none, routers of 1 to 16 experts, with
    and without feed-forward, embedding scale and soft cap."""
    import random
    rng = random.Random(seed)
    width = rng.choice([24, 48, 64, 96, 160])
    layers, lenders = [], []

    def mask():
        return rng.choice([1, 2, 9, 38, 63, 64, 65, 100, 1000]), rng.choice([0, 1, 2, 7, 63, 64, 65, 130])

    for i in range(rng.randint(2, 6)):
        kind = rng.choice(["retention", "attention", "attention"])
        if kind == "retention":
            h, d = rng.choice([1, 2, 3, 4]), rng.choice([4, 8, 16, 24, 32, 64, 128])
            rot = (rng.choice([100.0, 1e4, 1e6]), rng.choice(list(range(2, d + 1, 2)) + [d] * 3)) if rng.random() < 0.85 else None
            lay = ret(d, rng.choice([16 // h + 1, 8 + 4 * (h < 2), 16, 32, 48, 64, max(d, 16 // h + 1)]), [rng.choice([0.0, 0.5, 0.9, 0.97, 0.99, 0.999, 1.0]) for _ in range(h)], rot)
        else:
            if lenders and rng.random() < 0.45:
                src = rng.choice(lenders)
                m = layers[src][0]["mixer"]
                a, g, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            else:
                src = None
                g = rng.choice([1, 2, 3])
                a, d, dv = g * rng.choice([1, 2, 4]), rng.choice([2, 8, 16, 32, 48, 64, 128]), rng.choice([16 // g, 16, 24, 40, 64])
                if rng.random() < 0.4 and g * d >= 16:
                    dv = d
                lenders.append(i)
            lay = att(a, g, d, dv, rng.choice([0.1, d ** -0.5, 0.4]), *mask(), kv_from=src)
        mlp = rng.choice([None, "dense", "moe", "moe"])
        if mlp == "dense":
            mlp = dense(rng.choice([16, 20, 64, 100]))
        elif mlp == "moe":
            e = rng.choice([1, 2, 5, 8, 16])
            mlp = moe(e, rng.randint(1, min(e, 4)), rng.choice([12, 20, 32, 64]), rng.choice([0.2, 1.0, 7.0]))
        layers.append((lay, mlp))
    cfg = config(rng.choice([97, 256, 333]), width, rng.choice([1e-6, 1e-5]), rng.choice([1.0, 0.5, math.sqrt(width)]),
                 rng.choice([5.0, 25.0]), layers)
    if rng.random() < 0.2:
        del cfg["logit_softcap"]
    return cfg

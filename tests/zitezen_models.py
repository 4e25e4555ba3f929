"""Shared by the Zitezen tests: small configurations with sizes of their own, weights made here (larger
than the package's random fill, so that softmaxes are sharp and gates open and close), and model
folders written from them."""
import json
import math
import os
import struct
import tempfile

import torch

F32, BF16 = torch.float32, torch.bfloat16


def mem(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def mlstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": mem(heads, dim, vdim, cap)}


def lat(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
    return {"type": "latent_attention", "mixer": m}


def par(heads, kv_heads, dim, vdim, scale, cap, rot, left_scale, right, right_scale):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if cap:
        left["softcap"] = cap
    if rot:
        left["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": left_scale, "right": right, "right_scale": right_scale}}


def config(vocab, width, streams, eps, layers, loop=None):
    return {"architecture": "Zitezen", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)),
            "layers": [dict(lay, mlp=None if ff is None else {"kind": "dense", "ff": ff}) for lay, ff in layers]}


# odd sizes everywhere: a parallel layer first, a loop in the middle that repeats layers with and without
# feed-forward, three copies of the stream, key sizes above and below the value sizes, grouped and
# ungrouped key heads, rotation over part of a head, one cap that bites and one that hardly does
ZT_ODD = config(137, 42, 3, 3e-5, [
    (par(6, 2, 10, 14, 0.35, 3.0, (90.0, 6), 0.7, mem(3, 9, 5, 6.0), 1.4), 30),
    (mlstm(2, 7, 20, 4.0), 26),
    (lat(3, 10, 6, 14, 22, 18, 0.24, 700.0), None),
    (mlstm(5, 24, 6, 11.0), None),
    (par(3, 3, 12, 6, 0.28, 30.0, None, 1.2, mem(1, 20, 36, 9.0), 0.5), 44),
    (lat(4, 6, 4, 5, 16, 12, 0.3, 50.0), 20),
], loop=(1, 4, 2))
# sizes nearer to a served model's, taken by the tensor-core kernels: memories of 64 x 64, 128 x 96,
# 16 x 48 and 48 x 16, heads of 64 and 128 with grouped keys, two copies, a loop over the first two layers
ZT_WIDE = config(300, 128, 2, 1e-6, [
    (mlstm(2, 64, 64, 9.0), 192),
    (par(8, 2, 64, 64, 0.125, 12.0, (1e4, 32), 0.9, mem(3, 48, 16, 7.0), 1.2), None),
    (mlstm(1, 128, 96, 14.0), None),
    (lat(4, 32, 16, 48, 96, 64, 0.14, 1e5), 160),
    (par(2, 2, 128, 128, 0.09, 25.0, (1e5, 128), 1.1, mem(4, 16, 48, 12.0), 0.8), 96),
], loop=(0, 2, 3))
CONFIGS = {"odd": ZT_ODD, "wide": ZT_WIDE}


def tensor_shapes(cfg):
    """name -> (shape, kind) of every tensor of a Zitezen model, from its config alone."""
    w, s = cfg["width"], cfg["streams"]
    out = {"embed": ((cfg["vocab"], w), "table"), "head": ((cfg["vocab"], w), "matrix")}

    def norm(name):
        out.update({name: ((w,), "norm"), name + ".b": ((w,), "shift"), name + ".alpha": ((), "alpha")})

    def memory(q, m):
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        out.update({q + "q": ((H * d, w), "matrix"), q + "k": ((H * d, w), "matrix"), q + "v": ((H * dv, w), "matrix"),
                    q + "g": ((H * dv, w), "matrix"), q + "i": ((H, w), "gate"), q + "i.b": ((H,), "bias_i"), q + "f": ((H, w), "gate"),
                    q + "f.b": ((H,), "bias_f"), q + "norm": ((H * dv,), "norm"), q + "o": ((w, H * dv), "matrix")})

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        for j in ("1", "2") if layer["mlp"] else ("1",):
            norm(p + "norm" + j)
            out.update({p + "ls" + j: ((w,), "norm"), p + f"hc{j}.in": ((s,), "read"), p + f"hc{j}.out": ((s,), "write"),
                        p + f"hc{j}.mix": ((s, s), "mix")})
        if layer["type"] == "mlstm":
            memory(q, m)
        elif layer["type"] == "latent_attention":
            H, d, rd, dv, r, qr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            out.update({q + "dq": ((qr, w), "matrix"), q + "dq.norm": ((qr,), "norm"), q + "uq": ((H * (d + rd), qr), "matrix"),
                        q + "dkv": ((r + rd, w), "matrix"), q + "dkv.norm": ((r,), "norm"), q + "uk": ((H * d, r), "matrix"),
                        q + "uv": ((H * dv, r), "matrix"), q + "o": ((w, H * dv), "matrix")})
        else:
            a, q2 = m["left"], q + "left."
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            out.update({q2 + "q": ((H * d, w), "matrix"), q2 + "k": ((G * d, w), "matrix"), q2 + "v": ((G * dv, w), "matrix"),
                        q2 + "q.norm": ((d,), "norm"), q2 + "k.norm": ((d,), "norm"), q2 + "g": ((H, w), "matrix"),
                        q2 + "o": ((w, H * dv), "matrix")})
            memory(q + "right.", m["right"])
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({p + "mlp.up": ((ff, w), "matrix"), p + "mlp.down": ((w, ff), "matrix")})
    return out


def make_weights(cfg, seed, dt, steady=False):
    """``steady``: milder matrices, for the bfloat16 models.  The copies' matrices lie around a mixing that
    keeps their sizes; forget gates are mostly open, some far, so that the memory is long."""
    g = torch.Generator().manual_seed(seed)
    s, out = cfg["streams"], {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if kind == "norm":
            t = 1.0 + 0.2 * t
        elif kind == "alpha":
            t = 0.6 + 0.1 * t
        elif kind == "shift":
            t = 0.1 * t
        elif kind == "table":
            t = 0.8 * t
        elif kind == "gate":
            t = t * (1.5 / math.sqrt(shape[1]))
        elif kind == "bias_i":
            t = -1.0 + 1.5 * t
        elif kind == "bias_f":
            t = 4.0 + 1.5 * t
        elif kind == "read":
            t = 1.0 / s + 0.2 * t
        elif kind == "write":
            t = 0.6 + 0.3 * t
        elif kind == "mix":
            t = torch.eye(s) * 0.7 + 0.15 / s + 0.1 * t
        else:
            t = t * ((1.0 if steady else 1.6) / math.sqrt(shape[-1]))
        out[name] = t.to(dt)
    return out


def write_folder(cfg, weights):
    folder = tempfile.mkdtemp(prefix="bfi_zitezen_")
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, t in weights.items():
        raw = t.contiguous().reshape(-1).view(torch.int16 if t.dtype == BF16 else torch.int32).numpy().tobytes()
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
    """A configuration drawn from a seed: one to five layers of the three kinds in any order, sizes from
    lists that hold odd ones and values that make other sizes equal or 1, one to eight copies of the
    stream, loops over any range (also an empty one and a single pass), rotation over a whole head, a part
    of it or none, caps from tight to none, with and without feed-forward."""
    import random
    rng = random.Random(seed)
    width = rng.choice([24, 36, 64, 96, 160])

    def memory():
        h, d = rng.choice([1, 2, 3, 4]), rng.choice([1, 4, 8, 16, 24, 32, 48, 64, 128])
        return mem(h, d, rng.choice([max(2, 16 // h + 1), 16, 24, 32, 48, 64, max(d, 8)]), rng.choice([1.0, 4.0, 12.0, 15.0, 30.0]))

    layers = []
    for _ in range(rng.randint(1, 5)):
        kind = rng.choice(["mlstm", "latent", "parallel"])
        if kind == "mlstm":
            m = memory()
            lay = mlstm(m["heads"], m["dim"], m["vdim"], m["gate_cap"])
        elif kind == "latent":
            rd = rng.choice([0, 2, 4, 8, 16, 32])
            r = rng.choice([8, 14, 24, 32, 64, 128])
            d = rng.choice([1, 6, 16, 32, 64])
            lay = lat(rng.choice([1, 2, 3, 8]), d, rd, rng.choice([1 + 15 * (d == 1), 12, 16, 32, 64]), r, rng.choice([5, 16, 24, 64]),
                      rng.choice([0.12, (d + rd) ** -0.5]), rng.choice([30.0, 1e4, 1e6]))
        else:
            gk = rng.choice([1, 2, 3])
            d = rng.choice([2, 8, 16, 48, 64, 128])
            dv = d if rng.random() < 0.5 else rng.choice([16, 24, 40, 64])
            rot = (rng.choice([100.0, 1e4, 1e6]), rng.choice(list(range(2, d + 1, 2)) + [d] * 3)) if rng.random() < 0.85 else None
            lay = par(gk * rng.choice([1, 2, 4]), gk, d, max(dv, 16 // gk), rng.choice([0.1, d ** -0.5, 0.4]),
                      rng.choice([None, 0.5, 3.0, 20.0, 50.0]), rot, rng.choice([1.0, 0.8, 0.3]), memory(), rng.choice([1.0, 1.1, 2.0]))
        layers.append((lay, rng.choice([None, 16, 20, 64, 100])))
    loop = None
    if rng.random() < 0.7:
        a = rng.randint(0, len(layers) - 1)
        loop = (a, rng.randint(a, len(layers)), rng.choice([1, 2, 3]))
    return config(rng.choice([97, 256, 333]), width, rng.choice([1, 2, 3, 4, 5, 8]), rng.choice([1e-6, 1e-5]), layers, loop)

"""A plain, slow implementation of the Zitezen design: whole sequences, no cache, float64, one
function per mechanism, written from the design's equations and sharing nothing with the package.
The tests compare the package's kernels, parts and engine with it.

Notation: linear weights are ``[out, in]`` and act as ``W x``; ``w[name]`` is a tensor of the
checkpoint.  The residual stream is held ``s`` times, ``X`` ``[s, T, width]``, every copy the embedded
token at the start.  A sublayer (the mixer, and the feed-forward where the layer has one) reads a
weighted sum of the copies and is written back while the copies are mixed among themselves:

    u   = sum_a in[a] X_a
    y   = scale * sublayer(tanh(alpha u) w + b)            scale, w, b: one value per channel
    X_b = sum_a mix[a, b] X_a + out[b] y                   all copies from the old ones

The mixer is a matrix memory, latent attention, or soft-capped attention and a matrix memory side by
side; the feed-forward is ``W_down max(W_up h, 0)^2``.  The logits are ``head (tanh(alpha x) w + b)``
with ``x`` the sum of the copies.  A range of layers runs several times in a row.
"""
import json
import math
import os
import struct

import torch

F = torch.float64


# ------------------------------------------------------------------------------- files
def read_tensors(path):
    """name -> tensor of a safetensors file (8-byte length, JSON header, raw data)."""
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16}
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        blob = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        t = torch.frombuffer(bytearray(blob[a:b]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
        out[name] = t.to(F) if t.is_floating_point() else t
    return out


def load_folder(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_tensors(os.path.join(folder, "model.safetensors"))


# ------------------------------------------------------------------------------- small functions
def rms(x, eps):
    """x divided by its root mean square over the last dimension; eps sits inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def dynamic_tanh(x, alpha, weight, bias):
    return torch.tanh(alpha * x) * weight + bias


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def log_sigmoid(z):
    return torch.where(z >= 0, -torch.log1p(torch.exp(-z.abs())), z - torch.log1p(torch.exp(-z.abs())))


def squared_relu(z):
    return z.clamp(min=0.0) ** 2


# ------------------------------------------------------------------------------- rotation
def rotary_angles(positions, dims, base):
    """cos and sin ``[T, dims/2]`` of ``p * base^(-2i/dims)``."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=F) / dims)
    a = torch.tensor(list(positions), dtype=F)[:, None] * f[None, :]
    return torch.cos(a), torch.sin(a)


def rotate_halves(v, cos, sin, dims):
    """Of every head of ``v`` ``[T, heads, d]`` the first ``dims`` values, value i with value i + dims/2."""
    out, h = v.clone(), dims // 2
    a, b, c, s = v[..., :h], v[..., h:dims], cos[:, None, :], sin[:, None, :]
    out[..., :h], out[..., h:dims] = a * c - b * s, b * c + a * s
    return out


def rotate_neighbours(v, cos, sin, dims):
    """The same with value 2i and value 2i + 1."""
    out = v.clone()
    a, b, c, s = v[..., 0:dims:2], v[..., 1:dims:2], cos[:, None, :], sin[:, None, :]
    out[..., 0:dims:2], out[..., 1:dims:2] = a * c - b * s, b * c + a * s
    return out


# ------------------------------------------------------------------------------- softmax attention
def causal_attention(q, k, v, scale, cap=None):
    """``q`` ``[T, H, d]``, ``k`` ``[T, H, d]``, ``v`` ``[T, H, dv]``: every token over itself and all earlier
    ones; the scores soft-capped when ``cap`` is given."""
    T = q.shape[0]
    s = torch.einsum("iad,jad->aij", q, k) * scale
    if cap is not None:
        s = soft_cap(s, cap)
    future = torch.ones((T, T), dtype=torch.bool).triu(1)
    p = torch.softmax(s.masked_fill(future[None], float("-inf")), dim=-1)
    return torch.einsum("aij,jad->iad", p, v)


def attention(w, p, m, h, eps):
    """Grouped-query attention: norms per head before the rotation, soft-capped scores, one output
    gate per head."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T).view(T, H, d), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T).view(T, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(T, G, dv)
    rot = m.get("rot")
    if rot:
        cos, sin = rotary_angles(range(T), rot["dims"], rot["base"])
        q, k = rotate_halves(q, cos, sin, rot["dims"]), rotate_halves(k, cos, sin, rot["dims"])
    o = causal_attention(q, k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1), m["scale"], m.get("softcap"))
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def latent_attention(w, p, m, h, eps):
    """Queries through a normed latent; keys and values of all heads from one normed latent and one
    rotated key part that the heads share."""
    T = h.shape[0]
    H, d, rd, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T
    q = q.view(T, H, d + rd)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :r], eps) * w[p + "dkv.norm"]
    q_r, k_r = q[..., d:], down[:, r:].view(T, 1, rd)
    rot = m.get("rot")
    if rot:
        cos, sin = rotary_angles(range(T), rot["dims"], rot["base"])
        q_r, k_r = rotate_neighbours(q_r, cos, sin, rot["dims"]), rotate_neighbours(k_r, cos, sin, rot["dims"])
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), k_r.expand(T, H, rd)], dim=-1)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    o = causal_attention(torch.cat([q[..., :d], q_r], dim=-1), k, v, m["scale"])
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------- the matrix memory
def memory_scan(q, k, v, i, f, state=None):
    """One head, token by token: ``q``, ``k`` ``[T, d]``, ``v`` ``[T, dv]``, log gates ``i``, ``f`` ``[T]``.  ``state``
    ``(S, n, m)`` is what earlier tokens left (zeros at the start).  Returns ``o`` ``[T, dv]`` and the state."""
    S, n, m = state if state is not None else (torch.zeros((q.shape[1], v.shape[1]), dtype=F), torch.zeros(q.shape[1], dtype=F),
                                               torch.zeros((), dtype=F))
    rows = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + put * torch.outer(k[t], v[t])
        n = keep * n + put * k[t]
        m = new
        rows.append((S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(rows), (S, n, m)


def memory_gates(w, p, m, h):
    """The log input gate and log forget gate of every head, ``[T, heads]`` each."""
    cap = m["gate_cap"]
    i = soft_cap(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w[p + "f"].T + w[p + "f.b"], cap))
    return i, f


def matrix_memory(w, p, m, h, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).view(T, H, d), (h @ w[p + "v"].T).view(T, H, dv)
    i, f = memory_gates(w, p, m, h)
    heads = [memory_scan(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a])[0] for a in range(H)]
    o = torch.cat([rms(x, eps) for x in heads], dim=-1) * w[p + "norm"]
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------- the model
def mixer(w, p, layer, h, eps):
    m = layer["mixer"]
    if layer["type"] == "mlstm":
        return matrix_memory(w, p, m, h, eps)
    if layer["type"] == "latent_attention":
        return latent_attention(w, p, m, h, eps)
    if layer["type"] == "parallel":
        return m["left_scale"] * attention(w, p + "left.", m["left"], h, eps) \
            + m["right_scale"] * matrix_memory(w, p + "right.", m["right"], h, eps)
    raise ValueError(f"unknown layer type {layer['type']!r}")


def feed_forward(w, p, h):
    return squared_relu(h @ w[p + "up"].T) @ w[p + "down"].T


def connect(X, read, write, mix, fn):
    """One sublayer around the copies ``X`` ``[s, T, width]`` of the residual stream."""
    y = fn(torch.einsum("a,atw->tw", read, X))
    return torch.einsum("ab,atw->btw", mix, X) + write[:, None, None] * y[None]


def normed(w, name, x):
    return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])


def schedule(cfg):
    """The layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, w, tokens, keep_layers=False):
    """Logits ``[T, vocab]`` of one sequence (and, when asked, the sum of the copies after every layer run)."""
    eps = cfg["norm"]["eps"]
    X = w["embed"][list(tokens)][None].repeat(cfg["streams"], 1, 1)
    after = []
    for i in schedule(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        X = connect(X, w[p + "hc1.in"], w[p + "hc1.out"], w[p + "hc1.mix"],
                    lambda u: w[p + "ls1"] * mixer(w, p + "mix.", layer, normed(w, p + "norm1", u), eps))
        if layer.get("mlp") is not None:
            X = connect(X, w[p + "hc2.in"], w[p + "hc2.out"], w[p + "hc2.mix"],
                        lambda u: w[p + "ls2"] * feed_forward(w, p + "mlp.", normed(w, p + "norm2", u)))
        after.append(X.sum(dim=0))
    logits = normed(w, "final.norm", X.sum(dim=0)) @ w["head"].T
    return (logits, torch.stack(after)) if keep_layers else logits

"""A plain, slow implementation of the Zirivik design: whole sequences, no cache, float64, one
function per mechanism, written from the design's equations and sharing nothing with the package.
The tests compare the package's kernels, parts and engine with it.

Notation: ``x`` is the residual stream ``[T, width]``; ``h`` a normed copy of it; linear weights
are ``[out, in]`` and act as ``W x``; ``w[name]`` is a tensor of the checkpoint.

A layer is ``x += norm1b(mixer(norm1(x)))`` and, when it has a feed-forward,
``x += norm2b(ff(norm2(x)))``; every one of these norms multiplies by ``1 + weight``.
"""
import json
import math
import os
import struct

import torch

F = torch.float64
GATE_SLOPE = 1.702      # an expert's gate is g * sigmoid(1.702 g)


# ------------------------------------------------------------------------------- files
def read_tensors(path):
    """name -> tensor of a safetensors file (8-byte length, JSON header, raw data)."""
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}
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


# ------------------------------------------------------------------------------- norms
def rms(x, eps):
    """x divided by its root mean square over the last dimension; eps sits inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def offset_norm(x, weight, eps):
    """The block's norm: the weight is stored around zero and enters as 1 + weight."""
    return rms(x, eps) * (1.0 + weight)


# ------------------------------------------------------------------------------- retention
def rotate_half(x, positions, base, dims):
    """x [T, heads, d].  Of each head's first ``dims`` values, value i (i < dims/2) and value
    i + dims/2 form a pair that turns by the angle position * base^(-2i/dims); the rest pass."""
    half = dims // 2
    i = torch.arange(half, dtype=F)
    freq = torch.tensor(float(base), dtype=F) ** (-2.0 * i / dims)
    ang = torch.as_tensor(list(positions), dtype=F)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def decayed_recurrence(q, k, v, decay, state=None):
    """q, k [T, H, D]; v [T, H, V]; decay [H].  Per head S_t = decay_h S_(t-1) + k_t v_t^T and
    o_t = S_t^T q_t.  Returns o [T, H, V] and the last S."""
    T, H, D = q.shape
    V = v.shape[-1]
    S = torch.zeros(H, D, V, dtype=F) if state is None else state.clone()
    o = torch.zeros(T, H, V, dtype=F)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def retention_mixer(h, w, p, m, eps, first_position=0, state=None):
    """Returns the mixer's output and the state after the last token."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    pos = range(first_position, first_position + T)
    q = (h @ w[p + "q"].T).view(T, H, D)
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    rot = m.get("rot")
    if rot:
        q = rotate_half(q, pos, rot["base"], rot["dims"])
        k = rotate_half(k, pos, rot["base"], rot["dims"])
    o, S = decayed_recurrence(q, k * D ** -0.5, v, torch.tensor(m["decay"], dtype=F), state)
    g = h @ w[p + "g"].T
    y = rms(o, eps).reshape(T, H * V) * (g * torch.sigmoid(g))
    return y @ w[p + "o"].T, S


# ------------------------------------------------------------------------------- softmax attention
def window_mask(T, size=None, keep_first=0):
    """seen[i, j]: j <= i, and j is one of the last ``size`` positions or one of the first ``keep_first``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def masked_attention(q, k, v, scale, seen):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H/G)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        s = ((q[:, h] @ k[:, h // rep].T) * scale).masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out[:, h] = (e / e.sum(dim=-1, keepdim=True)) @ v[:, h // rep]
    return out


def attention_mixer(h, w, p, m, lent):
    """``lent``: the keys and values of the layer this one borrows from, or None.  Returns the output
    and the keys and values the layer used."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d)
    if lent is None:
        lent = ((h @ w[p + "k"].T).view(T, G, d), (h @ w[p + "v"].T).view(T, G, dv))
    mask = m.get("mask")
    seen = window_mask(T, mask["size"], mask.get("keep_first", 0)) if mask else window_mask(T)
    o = masked_attention(q, lent[0], lent[1], m["scale"], seen)
    return o.reshape(T, H * dv) @ w[p + "o"].T, lent


# ------------------------------------------------------------------------------- feed-forward
def dense_ff(h, w, p):
    """W_down relu(W_up h)^2."""
    return torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, router, top, report=None):
    """The chosen experts, best first, and their scores.  ``report`` collects the smallest distance
    between a chosen and an unchosen score."""
    s = torch.sigmoid(h @ router.T)
    best, idx = s.sort(dim=-1, descending=True, stable=True)
    if report is not None and s.shape[-1] > top:
        report.append(float((best[:, top - 1] - best[:, top]).min()))
    return idx[:, :top], best[:, :top]


def routed_ff(h, w, p, f, report=None):
    """The sum over the chosen experts of expert(score * h): the score scales an expert's input."""
    idx, s = route(h, w[p + "router"], f["router"]["top"], report)
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=F)
    for e in range(f["router"]["experts"]):
        for k in range(idx.shape[1]):
            rows = (idx[:, k] == e).nonzero().view(-1)
            if rows.numel():
                out[rows] += expert(h[rows] * s[rows, k][:, None], w, f"{p}e{e}.", f["expert"]["limit"])
    return out


# ------------------------------------------------------------------------------- the model
def forward(cfg, w, ids, layers=None, report=None):
    """Logits [T, vocab].  ``layers`` collects the residual stream after every layer, ``report`` the
    routers' smallest distances."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(list(ids))] * (cfg.get("embedding") or {}).get("scale", 1.0)
    lent = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = offset_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "retention":
            y, _ = retention_mixer(h, w, p + "mix.", m, eps)
        else:
            src = m.get("kv_from")
            y, lent[i] = attention_mixer(h, w, p + "mix.", m, None if src is None else lent[src])
        x = x + offset_norm(y, w[p + "norm1b"], eps)
        f = layer.get("mlp")
        if f is not None:
            h = offset_norm(x, w[p + "norm2"], eps)
            y = dense_ff(h, w, p + "mlp.") if f["kind"] == "dense" else routed_ff(h, w, p + "mlp.", f, report)
            x = x + offset_norm(y, w[p + "norm2b"], eps)
        if layers is not None:
            layers.append(x)
    logits = offset_norm(x, w["final.norm"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap")
    return logits if cap is None else cap * torch.tanh(logits / cap)


def greedy(cfg, w, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(forward(cfg, w, ids)[-1])))
    return ids[len(prompt):]

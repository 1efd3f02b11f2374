"""A plain, slow Dozetar: whole sequences, no cache, one function per mechanism.

It shares no code with the product path: it reads config.json and model.safetensors itself and computes with
ordinary tensor arithmetic, float64 by default so that it is the more exact side of every comparison. Notation:
T tokens, H query (or recurrent) heads, G key/value heads, dk the size of a query or key head, dv the size of a value
head, c the factor every sublayer's result is added with.

The design: x = table[id]; a layer is x <- x + c n1(mixer(x)), then, where it has a feed-forward, x <- x + c n2(ff(x)): a
sublayer reads the stream itself and its result is normed, n(y) = y / rms(y) w. A mixer is a matrix memory per head with
exponential gates kept in range by a running maximum; or two mixers side by side, windowed softmax attention (with the
first keys kept, a sink, biases, a norm of queries and keys over the whole projection) and linear attention with a fixed
decay per head, added with two fixed factors. The feed-forward is a choice of small squared-relu feed-forwards whose input
is scaled by the router's score. The logits are cap tanh(W n(x) / cap).
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np
import torch

_NP = {"F32": np.float32, "F64": np.float64, "F16": np.float16, "I32": np.int32, "I64": np.int64}

# the design adds this to the denominator of the matrix memory's read-out
DENOMINATOR_EPS = 1e-6

# None, or a dtype that stored activations are rounded to (what a 16-bit engine keeps between its kernels), so that a
# test can measure how far such rounding alone moves the logits of a model
ROUND = None


def kept(x):
    return x if ROUND is None else x.to(ROUND).to(x.dtype)


def read_folder(folder, dtype=torch.float64):
    """(config dict, {name: tensor}); floating tensors as ``dtype``, integer tables as int64."""
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    tensors = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        b, e = meta["data_offsets"]
        chunk = raw[8 + n + b:8 + n + e]
        if meta["dtype"] == "BF16":
            arr = (np.frombuffer(chunk, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)
        else:
            arr = np.frombuffer(chunk, dtype=_NP[meta["dtype"]])
        t = torch.from_numpy(arr.copy()).reshape(meta["shape"])
        tensors[name] = t.to(dtype) if t.is_floating_point() else t.to(torch.int64)
    return config, tensors


# ---------------------------------------------------------------- small pieces

def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def log_sigmoid(x):
    return -torch.log1p(torch.exp(-x.abs())) + torch.clamp(x, max=0.0)


def capped(x, cap):
    return cap * torch.tanh(x / cap)


def rotate_neighbours(x, positions, rot):
    """x [T, heads, d]: dimensions 2i and 2i + 1 of the first ``dims`` turn by position * base^(-2i / dims)."""
    dims = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    angle = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(angle)[:, None, :].to(x.dtype), torch.sin(angle)[:, None, :].to(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def visible(T, window=None, keep_first=0):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    see = j <= i
    if window is not None:
        see = see & ((i - j < window) | (j < keep_first))
    return see


def attend(q, k, v, scale, see, sink):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H * dv]. sink [H]: exp(sink) is one more term of the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    group = torch.arange(H) // (H // G)
    scores = torch.einsum("thd,shd->hts", q, k[:, group]) * scale
    scores = scores.masked_fill(~see[None], float("-inf"))
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(scores - top)
    total = e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top)
    return torch.einsum("hts,shd->thd", e / total, v[:, group]).reshape(T, -1)


# ---------------------------------------------------------------- mixers

def softmax_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    positions = torch.arange(T)
    q = kept(h @ w[p + "q"].T + w[p + "q.b"])
    k = kept(h @ w[p + "k"].T + w[p + "k.b"])
    v = kept(h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    q = (rms(q, eps) * w[p + "q.norm"]).reshape(T, H, dk)
    k = (rms(k, eps) * w[p + "k.norm"]).reshape(T, G, dk)
    q, k = kept(rotate_neighbours(q, positions, m["rot"])), kept(rotate_neighbours(k, positions, m["rot"]))
    mask = m.get("mask") or {}
    see = visible(T, mask.get("size"), mask.get("keep_first", 0))
    return kept(attend(q, k, v, m["scale"], see, w[p + "sink"])) @ w[p + "o"].T + w[p + "o.b"]


def decayed_recurrence(q, k, v, decay):
    """q, k [T, H, dk], v [T, H, dv], decay [H]: S <- decay S + k v^T from zero, o = S^T q; [T, H, dv]."""
    T, H, dk = q.shape
    S = q.new_zeros(H, dk, v.shape[2])
    out = q.new_zeros(T, H, v.shape[2])
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    return out


def linear_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(kept(h @ w[p + "q"].T)).reshape(T, H, dk)
    k = silu(kept(h @ w[p + "k"].T)).reshape(T, H, dk)
    v = silu(kept(h @ w[p + "v"].T)).reshape(T, H, dv)
    o = decayed_recurrence(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * dv)
    o = rms(o, eps) * w[p + "norm"] * torch.sigmoid(kept(h @ w[p + "g"].T))
    return kept(o) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    return m["left_scale"] * softmax_attention(h, w, p + "left.", m["left"], eps) + \
        m["right_scale"] * linear_attention(h, w, p + "right.", m["right"], eps)


def memory_gates(h, w, p, cap):
    """(log input gate, log forget gate), [T, H] each."""
    i = capped(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f = log_sigmoid(capped(h @ w[p + "f"].T + w[p + "f.b"], cap))
    return i, f


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, dk], v [T, H, dv], i, f [T, H] -> o [T, H, dv]. The memory S and the normalizer n hold everything divided
    by exp(M), M the running maximum, which starts at zero as they do."""
    T, H, dk = q.shape
    S, n, M = q.new_zeros(H, dk, v.shape[2]), q.new_zeros(H, dk), q.new_zeros(H)
    out = q.new_zeros(T, H, v.shape[2])
    for t in range(T):
        now = torch.maximum(f[t] + M, i[t])
        keep, take = torch.exp(f[t] + M - now), torch.exp(i[t] - now)
        M = now
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        weight = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-M)) + DENOMINATOR_EPS
        out[t] = torch.einsum("hij,hi->hj", S, q[t]) / weight[:, None]
    return out


def memory_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = kept(h @ w[p + "q"].T).reshape(T, H, dk) * dk ** -0.5
    k = kept(h @ w[p + "k"].T).reshape(T, H, dk)
    v = kept(h @ w[p + "v"].T).reshape(T, H, dv)
    i, f = memory_gates(h, w, p, m["gate_cap"])
    o = rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * dv)
    return kept(o * w[p + "norm"] * torch.sigmoid(kept(h @ w[p + "g"].T))) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward and model

def choose(h, router, top):
    """([T, top] expert numbers, [T, top] weights): the largest sigmoid scores, as scored."""
    score = torch.sigmoid(h @ router.T)
    best = torch.topk(score, top, dim=-1)
    return best.indices, best.values


def experts(h, w, p, m):
    chosen, weight = choose(h, w[p + "router"], m["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weight[t]):
            hidden = kept(torch.clamp(w[p + f"e{e}.up"] @ (s * h[t]), min=0.0) ** 2)
            out[t] += w[p + f"e{e}.down"] @ hidden
    return out


MIXERS = {"mlstm": memory_mixer, "parallel": side_by_side}


def forward(config, w, ids, return_layers=False):
    """Logits [T, vocab] of one whole sequence (and the stream after every layer)."""
    eps, c = config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(ids, dtype=torch.int64)]
    streams = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + c * rms(MIXERS[layer["type"]](kept(x), w, p + "mix.", layer["mixer"], eps), eps) * w[p + "norm1"]
        if layer.get("mlp") is not None:
            x = x + c * rms(experts(kept(x), w, p + "mlp.", layer["mlp"]), eps) * w[p + "norm2"]
        streams.append(x)
    logits = kept(rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = config.get("logit_softcap")
    if cap:
        logits = capped(logits, cap)
    return (logits, torch.stack(streams)) if return_layers else logits

"""A plain, slow Godotar: whole sequences, no cache, one function per mechanism.

It shares no code with the product path: it reads config.json and model.safetensors itself and computes with
ordinary tensor arithmetic, float64 by default so that it is the more exact side of every comparison. Notation:
T tokens, D model width, H heads, dk the size of a key (or receptance) head, dv of a value head.

The design: X = n(table[id]). The layers ``loop.start`` .. ``loop.stop - 1`` run ``loop.times`` times in a row; before
pass p row p of ``loop.step`` is added to the stream. A layer is x <- x + mixer(n1(x)) + ff(n2(x)), both norms over the
same x, n(x) = x / rms(x) * (1 + w). A mixer is a time mixer with a matrix state per head and a data-dependent decay per
key channel, or windowed attention over one latent row a token with a low-rank query and a gate per head. The
feed-forward is a silu gated unit, or experts chosen by a softmax router some of whose choices are the input itself, or
absent. The logits are scale * table . n(x).
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np
import torch

_NP = {"F32": np.float32, "F64": np.float64, "F16": np.float16, "I32": np.int32, "I64": np.int64}

SLOPE = 1.702                 # the design fixes the sigmoid's slope in an expert's unit

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


def norm(x, weight, eps):
    """The model's norm: its weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + weight)


def silu(x):
    return x * torch.sigmoid(x)


def shifted(h):
    """The row of the token before; zeros before the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)


def mix(h, weight):
    return h + (shifted(h) - h) * weight


def frequencies(rot):
    dims = rot["dims"]
    return float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: dimension i < dims / 2 pairs with i + dims / 2; the rest of a head passes unchanged."""
    dims = rot["dims"]
    half = dims // 2
    angle = positions.to(torch.float64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(angle)[:, None, :].to(x.dtype), torch.sin(angle)[:, None, :].to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(T, window=None):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    see = j <= i
    if window is not None:
        see = see & (i - j < window)
    return see


# ---------------------------------------------------------------- the time mixer

def decay(mixed, w, p):
    """The factor of every key channel's row of the state, per token: exp(-exp(.)), between 0 and 1."""
    return torch.exp(-torch.exp(kept(torch.tanh(mixed @ w[p + "w1"].T)) @ w[p + "w2"].T + w[p + "w0"]))


def recurrence(r, k, v, fade, u):
    """r, k, fade [T, H, dk], v [T, H, dv], u [H, dk] -> o [T, H, dv]: o_t = (S + diag(u) k v^T)^T r, then S <- diag(fade) S + k v^T."""
    T, H, dk = r.shape
    S = r.new_zeros(H, dk, v.shape[-1])
    out = torch.zeros_like(v)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t])
        S = fade[t][:, :, None] * S + kv
    return out


def time_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    r, k, v, g = (kept(kept(mix(h, w[p + "mu." + s])) @ w[p + s].T) for s in "rkvg")
    fade = decay(kept(mix(h, w[p + "mu.w"])), w, p)
    heads = lambda x: x.reshape(T, H, d)
    o = recurrence(heads(r), heads(k), heads(v), heads(fade), w[p + "u"])
    o = rms(o, eps).reshape(T, H * d) * w[p + "norm"]
    return kept(o * silu(g)) @ w[p + "o"].T


# ---------------------------------------------------------------- latent attention

def attend(q, k, v, scale, see):
    """q, k [T, H, d], v [T, H, dv] -> [T, H, dv]."""
    scores = torch.einsum("thd,shd->hts", q, k) * scale
    scores = scores.masked_fill(~see[None], float("-inf"))
    return torch.einsum("hts,shd->thd", torch.softmax(scores, dim=-1), v)


def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(T)
    cq = kept(rms(kept(h @ w[p + "dq"].T), eps) * w[p + "dq.norm"])
    q = kept(cq @ w[p + "uq"].T).reshape(T, H, d + dr)
    down = kept(h @ w[p + "dkv"].T)
    c = kept(rms(down[:, :R], eps) * w[p + "dkv.norm"])
    shared = kept(rotate_halves(down[:, None, R:], positions, m["rot"]))                  # one key part for all heads
    q = torch.cat([q[..., :d], kept(rotate_halves(q[..., d:], positions, m["rot"]))], dim=-1)
    k = torch.cat([(c @ w[p + "uk"].T).reshape(T, H, d), shared.expand(T, H, dr)], dim=-1)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    mask = m.get("mask")
    o = attend(q, k, v, m["scale"], visible(T, None if mask is None else mask["size"]))
    o = o * torch.sigmoid(kept(h @ w[p + "g"].T))[:, :, None]
    return kept(o.reshape(T, H * dv)) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forwards

def silu_unit(h, w, p):
    return kept(silu(kept(h @ w[p + "gate"].T)) * kept(h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p, limit):
    g = torch.clamp(kept(h @ w[p + "gate"].T), max=limit)
    u = torch.clamp(kept(h @ w[p + "up"].T), min=-limit, max=limit)
    return kept(g * torch.sigmoid(SLOPE * g) * (u + 1.0)) @ w[p + "down"].T


def choose(z, correction, top):
    """Router logits [T, outputs] -> (chosen [T, top] by falling corrected score, their weights): softmax scores, the choice by
    score + correction, the weights the chosen scores without it, divided by their sum."""
    s = torch.softmax(z, dim=-1)
    chosen = torch.topk(s + correction, top, dim=-1).indices
    weight = s.gather(-1, chosen)
    return chosen, weight / (weight.sum(-1, keepdim=True) + 1e-20)


def experts(h, w, p, f):
    r = f["router"]
    chosen, weight = choose(h @ w[p + "router"].T, w[p + "correction"], r["top"])
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        share = (weight * (chosen == e)).sum(-1, keepdim=True)
        rows = (share[:, 0] > 0).nonzero()[:, 0]
        if len(rows):
            y = h[rows] if e >= r["experts"] else expert(h[rows], w, f"{p}e{e}.", f["expert"]["limit"])
            out[rows] += share[rows] * y
    return out


# ---------------------------------------------------------------- the model

MIXERS = {"wkv": time_mixer, "latent_attention": latent_attention}


def feed_forward(h, w, p, f):
    return silu_unit(h, w, p) if f["kind"] == "dense" else experts(h, w, p, f)


def run_order(config):
    """[(layer, pass number if it is the first layer of a pass, else None)] in the order the layers run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(config, w, ids, return_layers=False):
    """Logits [T, vocab] of one whole sequence (and the stream after every layer run)."""
    eps = config["norm"]["eps"]
    x = norm(w["embed"][torch.as_tensor(ids, dtype=torch.int64)], w["embed.norm"], eps)
    streams = []
    for i, t in run_order(config):
        if t is not None:
            x = x + w["loop.step"][t]
        layer, p = config["layers"][i], f"l{i}."
        moved = MIXERS[layer["type"]](kept(norm(x, w[p + "norm1"], eps)) if layer["type"] != "wkv" else norm(x, w[p + "norm1"], eps),
                                      w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            moved = moved + feed_forward(kept(norm(x, w[p + "norm2"], eps)), w, p + "mlp.", layer["mlp"])
        x = x + moved
        streams.append(x)
    logits = (kept(norm(x, w["final.norm"], eps)) @ w["embed"].T) * config["logit_scale"]
    return (logits, torch.stack(streams)) if return_layers else logits

"""Small Dozetar configurations and random models for the tests; nothing here touches the disk unless asked."""
import copy

import torch

from damendaemon_b200.registry import architecture_of


def mlstm(heads, dim, vdim, cap):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def parallel(heads, kv_heads, dim, vdim, rot, mask, right, scales, scale=None):
    """rot: (dims, base); mask: (size, keep_first) or None; right: (heads, dim, vdim, decays)."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5,
            "rot": {"dims": rot[0], "base": rot[1]}}
    if mask is not None:
        left["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return "parallel", {"left": left, "right": dict(zip(("heads", "dim", "vdim", "decay"), right)), "left_scale": scales[0],
                        "right_scale": scales[1]}


def layer(mixer, moe=None):
    """moe: (experts, top, ff) or None."""
    mlp = None if moe is None else {"kind": "moe", "router": {"experts": moe[0], "top": moe[1]}, "expert": {"ff": moe[2]}}
    return {"type": mixer[0], "mixer": copy.deepcopy(mixer[1]), "mlp": mlp}


def model(vocab, width, layers, residual, cap=None, eps=1e-5):
    out = {"architecture": "Dozetar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": residual, "layers": layers}
    if cap is not None:
        out["logit_softcap"] = cap
    return out


# A: values larger than keys in the attention, smaller in both memories; half of a head rotated; a window of 20 (no multiple of
# a page) with three first keys; decays from fast to nearly none; a layer without a feed-forward; two and three experts a token
TINY_A = model(211, 64, [layer(parallel(4, 2, 16, 24, (8, 100.0), (20, 3), (3, 20, 12, [0.5, 0.97, 0.9999]), (1.3, 0.7)), (5, 2, 40)),
                         layer(mlstm(3, 24, 16, 5.0)),
                         layer(mlstm(1, 8, 40, 15.0), (7, 3, 24))], residual=0.9, cap=12.0)
# B: no cap on the logits; every head its own keys, heads rotated whole; a window smaller than a page and no first keys; no mask
# at all in the last layer, whose right factor is negative; one expert a token, and all of them; residual factor one
TINY_B = model(97, 48, [layer(parallel(3, 3, 8, 16, (8, 30.0), (7, 0), (1, 5, 9, [0.9]), (1.0, 1.0)), (4, 1, 20)),
                        layer(mlstm(2, 12, 20, 30.0), (4, 4, 16)),
                        layer(parallel(1, 1, 32, 32, (2, 77.0), None, (2, 8, 8, [0.0, 1.0]), (0.4, -1.5)))], residual=1.0, eps=1e-6)
# C: heads of 64 with keys of their own (what the tensor-core attention kernels take), 33 first keys behind a window of 100;
# memories of 64 by 64 and of 130 by 100
TINY_C = model(300, 256, [layer(mlstm(4, 64, 64, 8.0), (8, 2, 128)),
                          layer(parallel(4, 4, 64, 64, (32, 200000.0), (100, 33), (4, 64, 32, [0.6, 0.9, 0.99, 0.999]), (0.8, 0.3)), (6, 2, 64)),
                          layer(mlstm(2, 130, 100, 3.0))], residual=0.6, cap=25.0)
# D: awkward sizes: a width of 100, a vocabulary of 131, three query heads on a key/value head, keys of 20 and values of 12; more
# first keys than the window is long; memories with keys of 3 and 4; a window of one
TINY_D = model(131, 100, [layer(parallel(6, 2, 20, 12, (6, 50.0), (33, 40), (5, 3, 7, [0.3, 0.8, 0.95, 0.99, 0.5]), (0.9, 1.1)), (3, 2, 30)),
                          layer(mlstm(5, 4, 6, 6.0), (9, 1, 12)),
                          layer(parallel(2, 1, 12, 4, (12, 1000.0), (1, 1), (1, 33, 17, [0.95]), (0.5, 0.5)))], residual=0.8)
# E: head sizes that the padded prompt tiles take (40 and 104, one key/value head for four; 128), a memory with keys of 256
TINY_E = model(150, 128, [layer(parallel(4, 1, 40, 104, (16, 1000.0), (50, 2), (2, 128, 48, [0.9, 0.998]), (0.7, 0.6)), (4, 2, 56)),
                          layer(mlstm(2, 256, 24, 10.0), (5, 2, 40)),
                          layer(parallel(2, 2, 128, 128, (64, 300.0), (64, 65), (1, 16, 128, [0.97]), (0.5, 0.9)))], residual=0.5, cap=40.0)

CONFIGS = {"A": TINY_A, "B": TINY_B, "C": TINY_C, "D": TINY_D, "E": TINY_E}


def make_tensors(config, seed, sharpen=3.0, dtype=torch.float32, decided=False):
    """Random weights with the queries' norm weights scaled up, so that attention is peaky and a key that is wrongly seen or
    missed moves the logits; matrices rounded to ``dtype`` (the values a bfloat16 folder would hold). decided: the routers look at
    channels of the stream that hold well separated values per token and that no sublayer writes much to, so that no choice is
    close (rounding would decide a close one)."""
    arch = architecture_of(config)
    tensors = arch.random_tensors(arch.parse_config(config), seed, torch.float32)
    if decided:
        g = torch.Generator().manual_seed(seed + 1)
        E = max([layer["mlp"]["router"]["experts"] for layer in config["layers"] if layer["mlp"]])
        order = torch.rand(config["vocab"], E, generator=g).argsort(dim=1)
        tensors["embed"][:, :E] = torch.linspace(-2.0, 2.0, E)[order]
    for name, t in tensors.items():
        if name.endswith("q.norm"):
            tensors[name] = t * sharpen
        if decided and name.endswith((".norm1", ".norm2")):
            t[:E] *= 0.01
        if decided and name.endswith(".router"):
            t.mul_(0.02)
            t[:, :E] += torch.eye(t.shape[0], E)
    for name, t in tensors.items():
        if t.dim() == 2:
            tensors[name] = t.to(dtype).to(torch.float32)
    return tensors


def plain_tensors(tensors):
    return {k: v.double() for k, v in tensors.items()}


def random_requests(config, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, config["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}

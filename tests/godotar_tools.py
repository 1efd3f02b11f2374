"""Small Godotar configurations and random models for the tests; nothing here touches the disk unless asked."""
import copy

import torch

from damendaemon_b200.registry import architecture_of


def wkv(heads, dim, rank):
    return "wkv", {"heads": heads, "dim": dim, "decay_rank": rank}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, mask=None, base=10000.0, dims=None, scale=None):
    out = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
           "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": {"dims": dims or rot_dim, "base": base}}
    if mask is not None:
        out["mask"] = {"size": mask}
    return "latent_attention", out


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, identity, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": ff, "limit": limit}}


def layer(mixer, mlp):
    return {"type": mixer[0], "mixer": copy.deepcopy(mixer[1]), "mlp": copy.deepcopy(mlp)}


def model(vocab, width, layers, loop=None, scale=1.0, eps=1e-5):
    out = {"architecture": "Godotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# A: the second and third layer run three times; three heads of 16 with a decay of rank 6 (no multiple of 8); a window of 20
# (no multiple of a page), values smaller than keys, a latent of 24 + 8; two of five experts and three identity outputs
TINY_A = model(211, 64, [layer(wkv(3, 16, 6), dense(96)), layer(wkv(2, 24, 16), moe(5, 2, 3, 40, 0.9)),
                         layer(latent(3, 12, 8, 10, 24, 20, mask=20, base=300.0), moe(4, 3, 1, 24, 1.5))], loop=(1, 3, 3), scale=0.7)
# B: no loop; latent attention first, without a mask and without a feed-forward; one expert a token and no identity output;
# a window smaller than a page (7) on one head; a layer of time mixing alone; a logit scale above one
TINY_B = model(97, 48, [layer(latent(2, 16, 4, 24, 16, 40, base=50.0), None), layer(wkv(1, 24, 8), moe(5, 1, 0, 16, 3.0)),
                        layer(latent(1, 8, 2, 8, 14, 12, mask=7), dense(56)), layer(wkv(5, 8, 24), None)], scale=3.0, eps=1e-6)
# C: heads of 64 and sizes the tensor-core attention over latent rows takes (96 + 32; 64 + 16 with seventeen heads), windows of
# 100 and 33; the loop runs once (only its vector is added); four of eight experts and one identity output
TINY_C = model(300, 128, [layer(wkv(2, 64, 32), dense(256)), layer(latent(4, 64, 32, 64, 96, 64, mask=100), moe(8, 4, 1, 48, 2.5)),
                          layer(latent(17, 16, 16, 16, 64, 48, mask=33, base=100.0), None), layer(wkv(4, 32, 8), moe(6, 2, 2, 64, 1.0))],
               loop=(0, 2, 1), scale=0.5)
# D: awkward sizes: a width of 100, a vocabulary of 131, all layers in the loop, twice; heads of 20 with a decay of rank 5;
# part of the rotated part turned, a latent of 22 + 6, a window of 33; every one of three experts and two identity outputs
TINY_D = model(131, 100, [layer(wkv(3, 20, 5), moe(3, 5, 2, 30, 2.0)), layer(latent(6, 10, 6, 12, 22, 30, mask=33, base=77.0, dims=4), dense(52)),
                          layer(wkv(2, 12, 9), None)], loop=(0, 3, 2), scale=1.0)
# E: a head of 128 by 128; forty heads (more than a tile of single tokens holds) over rows of 136 + 24 with values of 8, a window
# of 50; mostly identity outputs
TINY_E = model(150, 192, [layer(latent(40, 8, 24, 8, 136, 32, mask=50, base=500.0), moe(2, 2, 6, 48, 4.0)), layer(wkv(1, 128, 16), dense(128)),
                          layer(wkv(2, 40, 8), moe(12, 3, 4, 32, 0.5))], loop=(1, 2, 2), scale=0.4)

CONFIGS = {"A": TINY_A, "B": TINY_B, "C": TINY_C, "D": TINY_D, "E": TINY_E}


def make_tensors(config, seed, sharpen=3.0, dtype=torch.float32, decided=False):
    """Random weights with the query latent's norm scaled up, so that attention is peaky and a key that is wrongly seen or missed
    moves the logits; matrices rounded to ``dtype`` (the values a bfloat16 folder would hold). decided: corrections so far
    apart that they alone choose the experts (a rounded activation then moves no choice; the weights still come from the
    scores)."""
    shuffle = torch.Generator().manual_seed(seed)
    arch = architecture_of(config)
    tensors = arch.random_tensors(arch.parse_config(config), seed, torch.float32)
    for name in tensors:
        if name.endswith("dq.norm"):
            tensors[name] = tensors[name] * sharpen
        if decided and name.endswith("correction"):
            tensors[name] = 2.0 * torch.randperm(tensors[name].numel(), generator=shuffle).float()
        t = tensors[name]
        if t.dim() == 2 and not name.endswith((".u", "loop.step")):
            tensors[name] = t.to(dtype).to(torch.float32)
    return tensors


def plain_tensors(tensors):
    return {k: (v.double() if v.is_floating_point() else v.long()) for k, v in tensors.items()}


def random_requests(config, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, config["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}

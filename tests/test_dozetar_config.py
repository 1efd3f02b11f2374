"""Dozetar's configuration, its description in parts, and the plain implementation's own pieces (CPU)."""
import copy
import math

import pytest
import torch

import plain_dozetar as plain
from dozetar_tools import CONFIGS, TINY_A, TINY_B, TINY_D, make_tensors, plain_tensors

from damendaemon_b200.config.reader import ConfigError
from damendaemon_b200.parts import cache_needs, tensor_decls
from damendaemon_b200.registry import architecture_of


def spec_of(config):
    arch = architecture_of(config)
    typed = arch.parse_config(config)
    return arch, typed, arch.build_spec(typed)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_configuration_round_trips_and_names_its_tensors(name):
    config = CONFIGS[name]
    arch, typed, spec = spec_of(config)
    assert typed.to_dict() == config
    assert arch.parse_config(typed.to_dict()) == typed
    wanted = set()
    for d in tensor_decls(spec):
        wanted |= {n for n, _ in d.pieces} if d.pieces else {d.name}
    tensors = arch.random_tensors(typed, 1)
    assert wanted == set(tensors)
    for d in tensor_decls(spec):
        for n, shape in (d.pieces or ((d.name, d.shape),)):
            assert tuple(tensors[n].shape) == tuple(shape), n


def test_states_and_pages_of_the_mixers():
    _, _, spec = spec_of(TINY_A)
    needs = cache_needs(spec)
    paged, memory = needs[0]
    assert (paged.kv_heads, paged.head_dim, paged.value_dim, paged.window, paged.keep_first) == (2, 16, 24, 20, 3)
    assert memory.shape == (3, 12, 32) and memory.name == ""
    # a gated memory keeps its normalizer as one more column, and the running maximum
    assert [(n.shape, n.name) for n in needs[1]] == [((3, 17, 32), ""), ((3,), "peak")]
    assert [(n.shape, n.name) for n in needs[2]] == [((1, 41, 8), ""), ((1,), "peak")]
    _, _, spec = spec_of(TINY_B)
    assert cache_needs(spec)[2][0].window is None and len(spec.layers[2].norms) == 1 and spec.head.softcap is None
    assert spec.layers[0].residual_factor == 1.0 and spec.layers[2].mixer.right_scale == -1.5


@pytest.mark.parametrize("change, message", [
    (lambda c: c.update(architecture="Other"), "architecture"),
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "share"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.9]), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.9, 1.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][2]["mlp"].update(kind="dense"), "moe"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=8), "experts a token"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
])
def test_bad_fields_are_refused(change, message):
    config = copy.deepcopy(TINY_A)
    change(config)
    with pytest.raises(ConfigError, match=message):
        architecture_of(config).parse_config(config)


def test_the_plain_memory_equals_its_explicit_sum():
    """Without the running maximum the memory is a plain weighted sum: S_t = sum_k exp(i_k + f_(k+1) + .. + f_t) k_k v_k^T, the
    read-out S^T q over max(|n . q|, 1) (everything the maximum divides by cancels, its start at zero included)."""
    g = torch.Generator().manual_seed(0)
    T, H, dk, dv = 9, 2, 3, 4
    q, k = (torch.randn(T, H, dk, dtype=torch.float64, generator=g) for _ in range(2))
    v = torch.randn(T, H, dv, dtype=torch.float64, generator=g)
    i = 2 * torch.randn(T, H, dtype=torch.float64, generator=g)
    f = plain.log_sigmoid(torch.randn(T, H, dtype=torch.float64, generator=g))
    o = plain.matrix_memory(q, k, v, i, f)
    for t in range(T):
        w = torch.stack([torch.exp(i[s] + f[s + 1:t + 1].sum(0)) for s in range(t + 1)])
        S = torch.einsum("sh,shi,shj->hij", w, k[:t + 1], v[:t + 1])
        n = torch.einsum("sh,shi->hi", w, k[:t + 1])
        below = torch.clamp((n * q[t]).sum(-1).abs(), min=1.0)
        want = torch.einsum("hij,hi->hj", S, q[t]) / below[:, None]
        assert torch.allclose(o[t], want, rtol=1e-4), t          # (the small number in the denominator is not scaled: 1e-6 off)
    decay = torch.tensor([0.5, 0.9], dtype=torch.float64)
    o = plain.decayed_recurrence(q, k, v, decay)
    want = sum(decay[:, None] ** (8 - s) * (k[s] * q[8]).sum(-1, keepdim=True) * v[s] for s in range(9))
    assert torch.allclose(o[8], want)


def test_the_plain_mask_and_router_by_hand():
    see = plain.visible(8, 3, 2)
    assert see[7].tolist() == [True, True, False, False, False, True, True, True]
    assert see[2].tolist() == [True] * 3 + [False] * 5 and plain.visible(4).tolist() == torch.ones(4, 4).tril().bool().tolist()
    h = torch.tensor([[1.0, 2.0]], dtype=torch.float64)
    router = torch.tensor([[1.0, 0.0], [0.0, 1.0], [-1.0, 0.0]], dtype=torch.float64)
    chosen, weight = plain.choose(h, router, 2)
    assert chosen.tolist() == [[1, 0]] and torch.allclose(weight, torch.sigmoid(torch.tensor([[2.0, 1.0]], dtype=torch.float64)))
    # the weight goes in squared: the input is scaled before the squared relu
    w = {"router": router, **{f"e{j}.up": torch.eye(2, dtype=torch.float64) for j in range(3)},
         **{f"e{j}.down": torch.eye(2, dtype=torch.float64) for j in range(3)}}
    out = plain.experts(h, w, "", {"router": {"top": 1}})
    s = 1 / (1 + math.exp(-2.0))
    assert torch.allclose(out, s * s * h ** 2)
    # a sink takes its share of a lone key's weight
    o = plain.attend(torch.zeros(1, 1, 2), torch.zeros(1, 1, 2), torch.ones(1, 1, 3), 1.0, plain.visible(1), torch.tensor([math.log(3.0)]))
    assert torch.allclose(o, torch.full((1, 3), 0.25))


def test_every_mechanism_moves_the_logits():
    """Leaving a mechanism out of the plain model changes its logits: none of them is idle in the test configurations."""
    config = TINY_A
    w = plain_tensors(make_tensors(config, 5))
    ids = torch.randint(0, config["vocab"], (40,), generator=torch.Generator().manual_seed(1)).tolist()
    base = plain.forward(config, w, ids)

    def moved(change=None, **new_w):
        other = copy.deepcopy(config)
        if change:
            change(other)
        return (plain.forward(other, {**w, **new_w}, ids) - base).abs().max().item()
    assert moved(lambda c: c.pop("logit_softcap")) > 1e-4
    assert moved(lambda c: c.update(residual_mult=1.0)) > 1e-3
    assert moved(lambda c: c["layers"][0]["mixer"]["left"].pop("mask")) > 1e-4
    assert moved(lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=2)) > 1e-4
    assert moved(lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=21)) > 1e-4
    assert moved(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=16)) > 1e-4
    assert moved(lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.97, 0.99])) > 1e-4
    assert moved(lambda c: c["layers"][0]["mixer"].update(right_scale=0.8)) > 1e-4
    assert moved(lambda c: c["layers"][1]["mixer"].update(gate_cap=6.0)) > 1e-4
    for name in ("l0.mix.left.q.b", "l0.mix.left.k.b", "l0.mix.left.v.b", "l0.mix.left.o.b", "l0.mix.left.sink", "l1.mix.i.b", "l1.mix.f.b"):
        assert moved(**{name: torch.zeros_like(w[name])}) > 1e-4, name
    assert moved(lambda c: c["layers"][2]["mlp"]["router"].update(top=2)) > 1e-4
    assert len(TINY_D["layers"]) == 3

"""Godotar's configuration, its description in parts, and the plain implementation's own pieces (CPU)."""
import copy

import pytest
import torch

import plain_godotar as plain
from godotar_tools import CONFIGS, TINY_A, TINY_B, TINY_C, TINY_D, make_tensors, plain_tensors

from damendaemon_b200.cache import PagedRows
from damendaemon_b200.config.reader import ConfigError
from damendaemon_b200.parts import cache_needs, tensor_decls
from damendaemon_b200.parts.positions import rotary_frequencies
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


def test_the_decay_rank_comes_from_the_tensors():
    config = copy.deepcopy(TINY_A)
    for entry in config["layers"]:
        entry["mixer"].pop("decay_rank", None)
    arch = architecture_of(config)
    typed = arch.parse_config(config)
    with pytest.raises(ValueError, match="rank"):
        arch.build_spec(typed)
    shapes = {"l0.mix.w1": (6, 64), "l1.mix.w1": (16, 64)}
    known = arch.sizes_from_shapes(typed, shapes)
    assert [l.mixer.decay_rank for l in known.layers[:2]] == [6, 16]
    assert known == arch.parse_config(TINY_A)
    with pytest.raises(ConfigError, match="decay_rank"):
        arch.sizes_from_shapes(typed, {"l0.mix.w1": (6, 64)})
    with pytest.raises(ConfigError, match="rows"):
        arch.sizes_from_shapes(arch.parse_config(TINY_A), {"l0.mix.w1": (7, 64)})
    # random weights for a configuration that names no rank choose one
    tensors = arch.random_tensors(typed, 3)
    assert tensors["l0.mix.w1"].shape[0] == tensors["l0.mix.w2"].shape[1] == 8


def test_the_run_order_repeats_the_loop_with_states_for_every_pass():
    _, _, spec = spec_of(TINY_A)
    assert [(e.layer, e.add_embedding, e.add_vector) for e in spec.run_order] == \
        [(0, False, None), (1, False, 0), (2, False, None), (1, False, 1), (2, False, None), (1, False, 2), (2, False, None)]
    needs = cache_needs(spec)
    assert len(needs) == len(spec.run_order)
    assert [n.name for n in needs[1]] == ["", "shift"] and needs[1][0].shape == (2, 24, 32) and needs[1][1].shape == (64,)
    assert needs[2] == [PagedRows(32, window=20)]
    assert plain.run_order(TINY_A) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None)]
    _, _, once = spec_of(TINY_C)
    assert [(e.layer, e.add_vector) for e in once.run_order] == [(0, 0), (1, None), (2, None), (3, None)]
    _, _, none = spec_of(TINY_B)
    assert [e.layer for e in none.run_order] == [0, 1, 2, 3] and none.pass_vectors is None
    assert cache_needs(none)[0] == [PagedRows(20)]                       # no mask: every key stays
    assert none.layers[0].kind == "pre_norm_mixer" and len(none.layers[0].norms) == 1
    assert len(none.layers[2].norms) == 2 and none.layers[2].kind == "parallel"


@pytest.mark.parametrize("change, message", [
    (lambda c: c.update(architecture="Other"), "architecture"),
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), "heads"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "rotated part"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "experts per token"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "dense"),
    (lambda c: c["loop"].update(stop=9), "run of the model"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
])
def test_bad_fields_are_refused(change, message):
    config = copy.deepcopy(TINY_A)
    change(config)
    with pytest.raises(ConfigError, match=message):
        architecture_of(config).parse_config(config)


def test_frequencies_equal_the_plain_ones():
    for config in CONFIGS.values():
        for built, raw in zip(spec_of(config)[2].layers, config["layers"]):
            if raw["type"] == "latent_attention":
                f, magnitude = rotary_frequencies(built.mixer.rotary)
                assert magnitude == 1.0 and torch.allclose(f, plain.frequencies(raw["mixer"]["rot"]), rtol=1e-14, atol=0)


def test_the_plain_recurrence_equals_its_explicit_sum():
    g = torch.Generator().manual_seed(0)
    r, k, v = (torch.randn(7, 2, 5, generator=g, dtype=torch.float64) for _ in range(3))
    fade = torch.rand(7, 2, 5, generator=g, dtype=torch.float64)
    u = torch.randn(2, 5, generator=g, dtype=torch.float64)
    out = plain.recurrence(r, k, v, fade, u)
    t, h = 6, 1
    want = sum(((r[t, h] * torch.prod(fade[j + 1:t, h], dim=0) * k[j, h]).sum()) * v[j, h] for j in range(t))
    want = want + (r[t, h] * u[h] * k[t, h]).sum() * v[t, h]
    assert torch.allclose(out[t, h], want, rtol=1e-12, atol=1e-12)
    assert torch.allclose(out[0, h], (r[0, h] * u[h] * k[0, h]).sum() * v[0, h])      # the first token sees the bonus only


def test_the_plain_router_by_hand():
    z = torch.log(torch.tensor([[0.1, 0.4, 0.3, 0.2]], dtype=torch.float64))
    none = torch.zeros(4, dtype=torch.float64)
    chosen, weight = plain.choose(z, none, 2)
    assert chosen.tolist() == [[1, 2]] and torch.allclose(weight, torch.tensor([[4 / 7, 3 / 7]], dtype=torch.float64))
    # the correction moves the choice, the weights are the scores without it
    chosen, weight = plain.choose(z, torch.tensor([0.5, 0.0, 0.0, 0.0], dtype=torch.float64), 2)
    assert chosen.tolist() == [[0, 1]] and torch.allclose(weight, torch.tensor([[0.2, 0.8]], dtype=torch.float64))
    # an identity output hands the input on
    w = {"router": torch.tensor([[0.0, 0.0], [0.0, 0.0], [5.0, 0.0]], dtype=torch.float64), "correction": torch.zeros(3, dtype=torch.float64)}
    h = torch.tensor([[3.0, -2.0]], dtype=torch.float64)
    f = {"router": {"experts": 2, "top": 1, "identity": 1}, "expert": {"ff": 1, "limit": 1.0}}
    assert torch.allclose(plain.experts(h, w, "", f), h)


def test_every_mechanism_moves_the_logits():
    """Leaving a mechanism out of the plain model changes its logits: none of them is idle in the test configurations."""
    config = TINY_A
    w = plain_tensors(make_tensors(config, 5))
    ids = torch.randint(0, config["vocab"], (40,), generator=torch.Generator().manual_seed(1)).tolist()
    base = plain.forward(config, w, ids)

    def moved(new_config=None, **new_w):
        return (plain.forward(new_config or config, {**w, **new_w}, ids) - base).abs().max().item()

    def changed(change):
        c = copy.deepcopy(config)
        change(c)
        return c
    assert moved(**{"loop.step": torch.zeros_like(w["loop.step"])}) > 1e-3
    assert moved(**{"embed.norm": torch.zeros_like(w["embed.norm"])}) > 1e-3
    for name in ("l0.mix.mu.r", "l0.mix.mu.k", "l1.mix.mu.v", "l1.mix.mu.g", "l1.mix.mu.w"):
        assert moved(**{name: torch.zeros_like(w[name])}) > 1e-4, name
    for name in ("l0.mix.u", "l0.mix.w0", "l1.mix.w2", "l1.mix.norm", "l1.norm2", "l2.mix.g", "l2.mix.dq.norm", "l2.mix.dkv.norm",
                 "l1.mlp.correction"):
        assert moved(**{name: torch.zeros_like(w[name])}) > 1e-4, name
    assert moved(changed(lambda c: c["loop"].update(times=2))) > 1e-3
    assert moved(changed(lambda c: c["layers"][2]["mixer"]["mask"].update(size=19))) > 1e-5
    assert moved(changed(lambda c: c["layers"][2]["mixer"].update(scale=0.1))) > 1e-4
    assert moved(changed(lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0.5))) > 1e-4
    assert moved(changed(lambda c: c["layers"][2]["mixer"]["rot"].update(base=200.0))) > 1e-5
    assert moved(changed(lambda c: c.update(logit_scale=0.6))) > 1e-2
    assert TINY_D["layers"][1]["mixer"]["rot"]["dims"] < TINY_D["layers"][1]["mixer"]["rot_dim"]

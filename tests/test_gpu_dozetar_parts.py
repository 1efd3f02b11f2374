"""Dozetar's kernels and parts, each alone against the plain implementation's function for the same mechanism."""
import math

import pytest
import torch

import plain_dozetar as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def layout(lengths, slots):
    """entry_start and entry_slot of a step whose entries bring ``lengths`` tokens."""
    return i32([sum(lengths[:j]) for j in range(len(lengths) + 1)]), i32(slots)


def cuts(total, sizes):
    out, at, i = [], 0, 0
    while at < total:
        n = min(sizes[i % len(sizes)], total - at)
        out.append((at, at + n))
        at, i = at + n, i + 1
    return out


class Sequences:
    """Two requests' projections and the states of a matrix memory, run through the kernels in any cutting."""

    def __init__(self, H, dk, dv, gated, dtype=torch.float32, total=57, cap=4.0, silu=False, scale=1.0):
        self.H, self.dk, self.dv, self.gated, self.cap, self.silu, self.scale, self.dtype = H, dk, dv, gated, cap, silu, scale, dtype
        self.width = 2 * H * dk + 2 * H * dv
        pad = -self.width % 8
        self.proj = {r: rnd(total - 9 * r, self.width + pad, seed=r).to(dtype) for r in range(2)}
        self.z = {r: rnd(total - 9 * r, 2 * H, seed=10 + r, scale=3.0) for r in range(2)}
        self.decay = torch.linspace(0.3, 0.999, H, dtype=torch.float64) if H > 1 else torch.tensor([0.9], dtype=torch.float64)
        self.fade = (1 - self.decay).float().to(DEV)
        self.weight = 1 + 0.1 * rnd(H * dv, seed=30)
        self.slot = {0: 3, 1: 1}
        self.eps, self.den_eps = 1e-5, 1e-6

    def pieces(self, p):
        a, b = self.H * self.dk, self.H * self.dv
        return p[:, :a], p[:, a:2 * a], p[:, 2 * a:2 * a + b], p[:, 2 * a + b:2 * a + 2 * b]

    def plain_read(self, r):
        q, k, v, _ = (t.double() for t in self.pieces(self.proj[r]))
        if self.silu:
            q, k, v = plain.silu(q), plain.silu(k), plain.silu(v)
        T, H = q.shape[0], self.H
        q, k, v = q.reshape(T, H, -1) * self.scale, k.reshape(T, H, -1), v.reshape(T, H, -1)
        if not self.gated:
            return plain.decayed_recurrence(q, k, v, self.decay)
        z = self.z[r].double()
        return plain.matrix_memory(q, k, v, plain.capped(z[:, :H], self.cap), plain.log_sigmoid(plain.capped(z[:, H:], self.cap)))

    def plain_out(self, r, together):
        o = self.plain_read(r)
        T = o.shape[0]
        o = plain.rms(o.reshape(T, -1) if together else o, self.eps).reshape(T, -1)
        return o * self.weight.double() * torch.sigmoid(self.pieces(self.proj[r])[3].double())

    def states(self):
        from damendaemon_b200 import kernels
        shape = kernels.memory_state_shape(self.H, self.dk, self.dv, self.gated)
        state = torch.full((4, *shape), float("nan"), device=DEV)
        peak = torch.full((4, self.H), float("nan"), device=DEV)
        for s in self.slot.values():
            state[s], peak[s] = 0, 0
        return state, peak

    def portion(self, parts, state, peak, together=False):
        """parts: [(request, from, to)] of one step; returns (the finished rows, the raw read-out)."""
        from damendaemon_b200 import kernels
        H, dk, dv = self.H, self.dk, self.dv
        p = torch.cat([self.proj[r][a:b] for r, a, b in parts]).to(DEV)
        z = torch.cat([self.z[r][a:b] for r, a, b in parts]).to(DEV)
        start, slots = layout([b - a for _, a, b in parts], [self.slot[r] for r, _, _ in parts])
        q, k, v, gate = self.pieces(p)
        fade, take, floor = self.fade, None, None
        if self.gated:
            fade, take, floor = kernels.memory_gates(z, self.cap, start, slots, peak)
        ops = kernels.memory_prepare(q, k, v, H, dk, dv, scale=self.scale, silu=self.silu, take=take)
        o = kernels.memory_scan(*ops, fade, start, slots, state, dk, dv)
        out = kernels.memory_finish(o, gate, self.weight.to(DEV), H, dv, self.eps, self.den_eps, floor=floor, together=together)
        return out, o

    def single(self, parts, state, peak, fused, slices=None, together=False):
        """A step of single tokens: parts [(request, position)]."""
        from damendaemon_b200 import kernels
        p = torch.cat([self.proj[r][t:t + 1] for r, t in parts]).to(DEV)
        z = torch.cat([self.z[r][t:t + 1] for r, t in parts]).to(DEV)
        q, k, v, gate = self.pieces(p)
        slots = i32([self.slot[r] for r, _ in parts])
        source = {"gates": (z, self.cap, peak)} if self.gated else {"fade": self.fade}
        sizes = (self.H, self.dk, self.dv)
        out = kernels.memory_step(q, k, v, gate, slots, state, *sizes, weight=self.weight.to(DEV) if fused else None, eps=self.eps,
                                  den_eps=self.den_eps, scale=self.scale, silu=self.silu, slices=slices, **source)
        if fused:
            return out
        return kernels.memory_finish(out[0], gate, self.weight.to(DEV), self.H, self.dv, self.eps, self.den_eps, floor=out[1],
                                     together=together)

    def run(self, parts, together=False):
        """parts: {request: [(from, to)]}, a step per index, the second request laid out first."""
        state, peak = self.states()
        out = {r: [] for r in self.proj}
        for i in range(max(len(p) for p in parts.values())):
            step = [(r, *parts[r][i]) for r in (1, 0) if i < len(parts[r])]
            got = self.portion(step, state, peak, together)[0].float().cpu()
            at = 0
            for r, a, b in step:
                out[r].append(got[at:at + b - a])
                at += b - a
        return {r: torch.cat(v) for r, v in out.items()}, state, peak


SIZES = [(3, 24, 16), (1, 5, 9), (2, 8, 8), (2, 12, 20), (4, 64, 64), (2, 130, 100), (5, 3, 7), (2, 256, 24), (1, 33, 200), (3, 1, 1), (2, 16, 600)]


@pytest.mark.parametrize("gated", [True, False])
@pytest.mark.parametrize("H, dk, dv", SIZES)
def test_the_memory_in_portions_with_shuffled_slots(H, dk, dv, gated):
    """Two requests in portions down to one token beside each other, in slots that are not in order, against the plain
    recurrence, normed per head and together; a prompt cut anywhere gives the same bits as the prompt whole."""
    s = Sequences(H, dk, dv, gated, silu=not gated, scale=dk ** -0.5 if gated else 1.0)
    total = 57
    for together in (False, True):
        whole, state, peak = s.run({0: [(0, total)], 1: [(0, total - 9)]}, together)
        cut, state2, peak2 = s.run({0: cuts(total, (1, 2, 7, 1, 1, 16)), 1: cuts(total - 9, (5, 1, 1, 30))}, together)
        for r in (0, 1):
            # a first token's read-out may nearly vanish before it is divided by its root mean square
            want = s.plain_out(r, together)
            assert torch.allclose(whole[r].double(), want, atol=2e-3, rtol=1e-3), (r, (whole[r].double() - want).abs().max())
            assert (whole[r].double() - want).abs().mean() < 2e-5
            assert torch.equal(whole[r], cut[r])
        for slot in s.slot.values():
            assert torch.equal(state[slot], state2[slot]) and (not gated or torch.equal(peak[slot], peak2[slot]))
        assert torch.isnan(state[0]).all() and torch.isnan(state[2]).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("gated", [True, False])
@pytest.mark.parametrize("H, dk, dv, slices", [(3, 24, 16, (1, 2, 8)), (1, 5, 9, (1, 4)), (4, 64, 64, (1, 4)), (2, 130, 100, (1, 2, 8)),
                                               (5, 3, 7, (1, 4)), (2, 256, 24, (1, 8)), (2, 16, 600, (1, 8)), (3, 1, 1, (1,))])
def test_single_tokens_in_one_kernel(H, dk, dv, slices, gated, dtype):
    """Steps of single tokens after a prompt, with a head's columns cut over one to eight blocks of a cluster, fused with the norm
    and not: the states keep the bits of the same tokens run as portions, the rows are theirs up to the order of a sum."""
    s = Sequences(H, dk, dv, gated, dtype, silu=not gated, scale=dk ** -0.5 if gated else 1.0)
    tol = 3e-3 if dtype == torch.float32 else 0.05
    for n in slices:
        for fused in (True, False):
            state, peak = s.states()
            state2, peak2 = s.states()
            for st, pk in ((state, peak), (state2, peak2)):
                s.portion([(1, 0, 6), (0, 0, 4)], st, pk)
            for i in range(12):
                got = s.single([(0, 4 + i), (1, 6 + i)], state, peak, fused, n)
                want, _ = s.portion([(0, 4 + i, 5 + i), (1, 6 + i, 7 + i)], state2, peak2)
                assert (got.float() - want.float()).abs().max() < tol, (n, fused, i)
                plain_rows = torch.stack([s.plain_out(0, False)[4 + i], s.plain_out(1, False)[6 + i]])
                assert (got.cpu().double() - plain_rows).abs().mean() < (1e-4 if dtype == torch.float32 else 1e-2)
            for slot in s.slot.values():
                assert torch.equal(state[slot], state2[slot]), (n, fused)
                assert not gated or torch.equal(peak[slot], peak2[slot])
        together = s.single([(0, 30)], *s.states(), False, n, together=True)
        assert torch.isfinite(together).all()


def test_the_running_maximum_where_gates_are_extreme():
    """Input gates from far below to far above everything before (the maximum stays at its start, zero, then jumps), forget gates
    that drop everything and that drop nothing: the read-out, whose denominator is now the normalizer and now exp(-M), follows
    the plain memory, and nothing overflows."""
    for seed in range(3):
        s = Sequences(2, 8, 8, True, total=40, cap=40.0)
        for r in (0, 1):
            z = s.z[r]
            z[:] = rnd(*z.shape, seed=50 + seed + r, scale=30.0)
            z[:8, :2] = -60.0                             # the first tokens barely enter: the maximum stays at zero
            z[8, :2] = 80.0                               # and jumps here
            z[12:20, 2:] = 90.0                           # nothing is forgotten
            z[20, 2:] = -90.0                             # everything is
        want = {r: s.plain_read(r) for r in (0, 1)}
        state, peak = s.states()
        out, o = s.portion([(1, 0, 31), (0, 0, 40)], state, peak)
        assert torch.isfinite(out).all()
        from damendaemon_b200 import kernels
        start, slots = layout([31, 40], [1, 3])
        fresh = torch.zeros(4, 2, device=DEV)
        z = torch.cat([s.z[1], s.z[0]]).to(DEV)
        fade, take, floor = kernels.memory_gates(z, s.cap, start, slots, fresh)
        assert (take <= 1.0).all() and (fade <= 1.0).all() and (fade > -4e-6).all()      # (half a spacing of the floats near the maximum)
        o = o.view(71, 2, -1)
        read = o[:, :, :8] / (torch.maximum(o[:, :, 8].abs(), floor) + 1e-6)[:, :, None]
        plain_rows = torch.cat([want[1], want[0]])
        err = (read.cpu().double() - plain_rows).abs().amax(-1)
        assert (err <= 1e-4 * plain_rows.abs().amax(-1).clamp(min=1.0)).all(), err.max()


@pytest.mark.parametrize("gated", [True, False])
def test_a_token_far_back_reaches_the_read_out_through_a_slow_memory(gated):
    """A head that hardly forgets carries one marked token over 3,000 steps although what it loses per step is 1e-5: to a relative
    2e-5 with a fixed decay (one kept as a float32 number near one would be off by 1e-4 at the end), to 2e-4 with gates, where what
    the running maximum loses to rounding at every step (half a spacing of the floats near five, 7e-4 over the distance) must come
    back in the fade."""
    from damendaemon_b200 import kernels
    T, dk, dv = 3000, 4, 4
    q, k, v = torch.zeros(T, dk), torch.zeros(T, dk), torch.zeros(T, dv)
    q[:, 0] = 1.0
    k[0, 0] = 1.0
    v[0] = torch.tensor([1.0, -2.0, 3.0, 0.5])
    start, slots = layout([T], [0])
    buffer = torch.cat([q, k, v], dim=1).to(DEV)
    q, k, v = buffer[:, :dk], buffer[:, dk:2 * dk], buffer[:, 2 * dk:]
    state = torch.zeros(1, *kernels.memory_state_shape(1, dk, dv, gated), device=DEV)
    lost = 9.775e-6 if gated else 1e-5                   # 20.5 spacings of the floats near five
    if gated:
        cap = 20.0
        z = torch.full((T, 2), -20.0)                    # f = log sigmoid(c) = -lost at c = -log(expm1(lost))
        z[:, 1] = cap * math.atanh(-math.log(math.expm1(lost)) / cap)
        z[0, 0] = 20.0 * math.atanh(5.0 / 20.0)          # the marked token lifts the maximum to 5
        peak = torch.zeros(1, 1, device=DEV)
        fade, take, floor = kernels.memory_gates(z.to(DEV), cap, start, slots, peak)
        f = plain.log_sigmoid(plain.capped(z[:, 1].double(), cap))
        i = plain.capped(z[:, :1].double(), cap)
        M, total = torch.zeros(1, dtype=torch.float64), 0.0
        for t in range(T):
            total += float(f[t])
        # S_T exp(M_T) = exp(i_0 + the sum of f behind it), whatever the maximum did
        ops = kernels.memory_prepare(q, k, v, 1, dk, dv, take=take)
        o = kernels.memory_scan(*ops, fade, start, slots, state, dk, dv)
        got = o[-1, 0, :dv].cpu().double() * math.exp(float(peak[0, 0])) / math.exp(float(i[0, 0]))
        want = v[0].cpu().double() * math.exp(total - float(f[0]))
        assert torch.allclose(got, want, rtol=2e-4, atol=1e-6), (got / want)
    else:
        fade = torch.tensor([lost], dtype=torch.float64).float().to(DEV)
        ops = kernels.memory_prepare(q, k, v, 1, dk, dv)
        o = kernels.memory_scan(*ops, fade, start, slots, state, dk, dv)
        want = v[0].cpu().double() * (1 - lost) ** (T - 1)
        assert torch.allclose(o[-1, 0, :dv].cpu().double(), want, rtol=2e-5, atol=0)


@pytest.mark.parametrize("H, dv", [(3, 16), (2, 600), (5, 7), (1, 1), (9, 512), (4, 1100)])
def test_the_read_outs_norm(H, dv):
    """Per head and over all heads together, with and without a denominator, at widths that stay in registers and beyond."""
    from damendaemon_b200 import kernels
    n = 5
    for floor in (None, torch.exp(rnd(n, H, seed=1))):
        row = -(-(dv + (floor is not None)) // 4) * 4
        o = rnd(n, H, row, seed=2, scale=3.0)
        gate, weight = rnd(n, H * dv + 8, seed=3), 1 + 0.1 * rnd(H * dv, seed=4)
        x = o[:, :, :dv].double()
        if floor is not None:
            x = x / (torch.maximum(o[:, :, dv].abs(), floor).double() + 1e-6)[:, :, None]
        for together in (False, True):
            y = plain.rms(x.reshape(n, -1) if together else x, 1e-5).reshape(n, -1)
            for dtype in (torch.float32, torch.bfloat16):
                g = gate.to(dtype).to(DEV)[:, 4:4 + H * dv]
                want = y * weight.double() * torch.sigmoid(g.cpu().double())
                got = kernels.memory_finish(o.to(DEV), g, weight.to(DEV), H, dv, 1e-5, 1e-6, floor=None if floor is None else floor.to(DEV),
                                            together=together)
                assert got.dtype == dtype
                assert (got.cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 0.05)


@pytest.mark.parametrize("width", [40, 100, 101, 1024, 1600, 2048, 4096, 5000, 7001])
def test_a_result_normed_and_added_to_the_stream(width):
    """One result, two with factors, and the sum of a token's rows; with the norm and without; the rounded copy is the stream's."""
    from damendaemon_b200 import kernels
    n, top = 6, 5
    x, a, b = rnd(n, width, seed=1), rnd(n, width, seed=2, scale=5.0), rnd(n, width, seed=3, scale=0.1)
    w, rows = 1 + 0.1 * rnd(width, seed=4), rnd(20, width, seed=5)
    pair = torch.randint(0, 20, (n * top,), generator=torch.Generator().manual_seed(6)).to(torch.int32)
    pair[3] = -1                                          # no row
    picked = torch.stack([sum(rows[r].double() for r in pair[t * top:(t + 1) * top].tolist() if r >= 0) for t in range(n)])
    cases = [({"a": a.to(DEV)}, a.double()),
             ({"a": a.to(DEV), "scale": 0.3, "other": b.to(DEV), "other_scale": -2.0}, 0.3 * a.double() - 2.0 * b.double()),
             ({"a": rows.to(DEV), "pair_row": pair.to(DEV)}, picked)]
    for terms, y in cases:
        want = x.double() + 0.9 * plain.rms(y, 1e-5) * w.double()
        for dtype in (None, torch.bfloat16):
            stream = x.to(DEV).clone()
            low = kernels.post_norm(stream, weight=w.to(DEV), eps=1e-5, factor=0.9, rounded_dtype=dtype, **terms)
            assert torch.allclose(stream.cpu().double(), want, atol=1e-5)
            assert low is None if dtype is None else torch.equal(low, stream.to(torch.bfloat16))
        stream = x.to(DEV).clone()
        kernels.post_norm(stream, factor=0.9, **terms)
        assert torch.allclose(stream.cpu().double(), x.double() + 0.9 * y, atol=1e-5)
    assert torch.equal(kernels.round_rows(x.to(DEV), torch.bfloat16), x.to(DEV).to(torch.bfloat16))
    assert kernels.round_rows(stream, torch.float32) is stream


@pytest.mark.parametrize("dtype, width, ff", [(torch.float32, 40, 24), (torch.bfloat16, 64, 40), (torch.bfloat16, 256, 136),
                                              (torch.bfloat16, 100, 30), (torch.float32, 33, 7)])
@pytest.mark.parametrize("experts, top, tokens", [(5, 1, 37), (4, 4, 9), (12, 3, 150), (1, 1, 3)])
def test_experts_whose_input_is_weighted(experts, top, tokens, dtype, width, ff):
    """The part against the plain experts: as terms of a norm and added to a stream, on the tensor cores and beside them (widths
    that are no multiple of eight)."""
    from damendaemon_b200 import kernels
    from damendaemon_b200.parts.feed_forward import ScoreRoutedExperts
    from damendaemon_b200.parts.interfaces import Runtime
    from damendaemon_b200.parts.spec import PlainUnitSpec, ScoreRoutedExpertsSpec
    units = tuple(PlainUnitSpec(ff, f"e{j}.up", f"e{j}.down", "relu2") for j in range(experts))
    spec = ScoreRoutedExpertsSpec("experts_by_score", width=width, top=top, router="router", experts=units, weight_input=True)
    w = {"router": rnd(experts, width, seed=1)}
    for j in range(experts):
        w[f"e{j}.up"], w[f"e{j}.down"] = rnd(ff, width, seed=10 + j) / width ** 0.5, rnd(width, ff, seed=30 + j) / ff ** 0.5
    w = {n: t.to(dtype) for n, t in w.items()}
    h = rnd(tokens, width, seed=2).to(dtype)
    want = plain.experts(h.double(), {n: t.double() for n, t in w.items()}, "", {"router": {"top": top}})
    part = ScoreRoutedExperts(spec, {n: t.to(DEV) for n, t in w.items()}, Runtime(dtype=dtype, device=torch.device(DEV)))
    assert part.tensor_cores == (dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0)
    tol = (1e-4 if dtype == torch.float32 else 0.02) * max(1.0, want.abs().max().item())
    stream = torch.zeros(tokens, width, device=DEV)
    kernels.post_norm(stream, **part.forward_terms(h.to(DEV), None))
    assert (stream.cpu().double() - want).abs().max() < tol
    x = rnd(tokens, width, seed=3)
    assert (part.forward(h.to(DEV), x.to(DEV).clone(), None).cpu().double() - x.double() - want).abs().max() < tol
    assert (part.forward(h.to(DEV), None, None).cpu().double() - want).abs().max() < tol
    assert kernels.read_error_flag(DEV) == 0


def test_sorted_rows_carry_their_weights():
    from damendaemon_b200 import kernels
    n, top, E, tile = 70, 3, 6, 16
    g = torch.Generator().manual_seed(0)
    table = torch.rand(n, E, generator=g).argsort(1)[:, :top].to(torch.int32).contiguous()
    weight = torch.rand(n * top, generator=g) + 0.1
    pair_row, row_token, tile_group, row_weight = kernels.route_by_table(None, table.to(DEV), E, tile, pair_weight=weight.to(DEV))
    assert torch.equal(row_weight[pair_row.long()].cpu(), weight)
    assert (row_weight[row_token < 0] == 0).all() and (row_token[pair_row.long()].cpu() == torch.arange(n).repeat_interleave(top)).all()
    assert torch.equal(tile_group[(pair_row // tile).long()].cpu(), table.reshape(-1))


def paged(k, v, page, seed):
    """Keys [T, G, dk] and values [T, G, dv] of one sequence in shuffled pages of a poisoned cache: (cache, block table)."""
    from damendaemon_b200 import kernels
    (T, G, dk), dv = k.shape, v.shape[2]
    used = -(-T // page)
    pages = torch.randperm(used + 3, generator=torch.Generator().manual_seed(seed))[:used].tolist()
    table = i32([pages + [-1] * 3])
    shape = (used + 3, 2, G, page, dk) if dk == dv else (used + 3, G * page * (dk + dv))
    cache = torch.full(shape, float("nan"), dtype=k.dtype, device=DEV)
    buffer = torch.cat([k.reshape(T, -1), v.reshape(T, -1)], dim=1).to(DEV)
    kernels.kv_store(buffer[:, :G * dk], buffer[:, G * dk:], i32([0] * T), i32(list(range(T))), table, cache, kv_heads=G, head_dim=dk, v_dim=dv)
    return cache, table


@pytest.mark.parametrize("H, G, dk, dv, window, keep", [(4, 1, 40, 104, 50, 2), (6, 2, 112, 56, 70, 5), (2, 2, 16, 8, 33, 40), (3, 1, 128, 56, None, 0),
                                                        (2, 2, 72, 72, 64, 64), (5, 5, 8, 128, 1, 1), (4, 2, 64, 24, 130, 0)])
def test_prompt_attention_in_padded_tiles(H, G, dk, dv, window, keep):
    """Head sizes the prompt kernel takes in padded tiles, in bfloat16: whole prompts, portions that start anywhere and single
    tokens against the plain attention with a sink and kept first keys; with the weights in two terms the rows are the general
    kernel's."""
    from damendaemon_b200 import kernels
    T, page = 330, 16
    bf = lambda t: t.to(torch.bfloat16)
    q, k, v = bf(rnd(T, H, dk, seed=1)), bf(rnd(T, G, dk, seed=2)), bf(rnd(T, G, dv, seed=3))
    sink, scale = rnd(H, seed=4), 2.0 * dk ** -0.5
    want = plain.attend(q.double(), k.double(), v.double(), scale, plain.visible(T, window, keep), sink.double())
    cache, table = paged(k, v, page, 5)
    assert kernels.attention_prefill_padded_supported(H, G, dk, dv, torch.bfloat16)
    sizes = {} if dk == dv else dict(kv_heads=G, v_dim=dv)
    kw = dict(window=window, keep_first=keep, sink=sink.to(DEV), **sizes)
    qd = q.reshape(T, -1).to(DEV)
    rows = kernels.attention_rows(qd, cache, i32([0] * T), i32(list(range(T))), table, H, scale, **kw)
    for exact in (False, True):
        tol = 0.012 if exact else 0.03
        for first, n in ((0, T), (0, 1), (1, 2), (63, 66), (64, 64), (129, 201), (T - 1, 1), (200, 65)):
            part = kernels.attention_prefill_padded(qd[first:first + n], cache, i32([0, n]), i32([first]), table, H, scale,
                                                    exact_weights=exact, **kw)
            assert part.shape == (n, H * dv) and (part.cpu().double() - want[first:first + n]).abs().max() < tol, (exact, first, n)
            if exact:
                assert (part.float() - rows[first:first + n].float()).abs().max() <= 2.0 ** -7 * max(1.0, rows.float().abs().max().item())
    assert kernels.read_error_flag(DEV) == 0


@pytest.mark.parametrize("dk, dv", [(40, 104), (112, 56), (16, 16)])
@pytest.mark.parametrize("window, keep", [(40, 20), (16, 3), (7, 9), (33, 0), (64, 64), (65, 130)])
def test_a_marked_key_at_every_edge_decides_the_output_of_the_padded_tiles(window, keep, dk, dv):
    """One key that the query matches a hundred times better than the rest: the output is its value exactly where the mask lets it
    through; just inside and outside the window and the kept keys, at tile borders, far away, at the query's own place."""
    from damendaemon_b200 import kernels
    H, page = 2, 16
    for pos in (window + keep + 30, 199, 64, 300):
        edges = {pos - window + 1, pos - window, pos - window + 2, pos, 0, keep - 1, keep, 63, 64, 127}
        for marked in sorted(m for m in edges if 0 <= m <= pos):
            seen = pos - marked < window or marked < keep
            T = pos + 1
            k, v, q = rnd(T, 1, dk, seed=1) * 0.1, rnd(T, 1, dv, seed=2) * 0.1, rnd(T, H, dk, seed=3) * 0.1
            k[marked], q[pos] = 0.0, 0.0
            k[marked, :, 3], q[pos, :, 3] = 30.0, 30.0
            v[marked] = torch.arange(dv) % 16 + 5.0
            cache, table = paged(k.to(torch.bfloat16), v.to(torch.bfloat16), page, marked)
            qd = q.reshape(T, -1).to(torch.bfloat16).to(DEV)
            first = max(0, pos - 69)
            out = kernels.attention_prefill_padded(qd[first:], cache, i32([0, T - first]), i32([first]), table, H, 1.0, window=window,
                                                   keep_first=keep, sink=torch.zeros(H, device=DEV), exact_weights=True,
                                                   **({} if dk == dv else dict(kv_heads=1, v_dim=dv)))[-1]
            hit = (out.float().cpu().view(H, dv) - v[marked]).abs().max().item() < 0.3
            assert hit == seen, (pos, marked, seen)


def test_neighbouring_pairs_turn_after_a_norm_over_the_whole_projection():
    """Queries and keys normed over all heads at once, then the first dimensions of every head turned in neighbouring pairs, at
    positions up to 5,000."""
    from damendaemon_b200 import kernels
    for H, G, d, dims in ((4, 2, 16, 8), (3, 1, 20, 20), (6, 2, 72, 40), (2, 2, 40, 2)):
        rot = {"dims": dims, "base": 500.0}
        positions = torch.tensor([0, 1, 7, 400, 4999])
        buffer = rnd(5, (H + G) * d + 8, seed=1, scale=2.0)
        wq, wk = 1 + 0.1 * rnd(H * d, seed=2), 1 + 0.1 * rnd(G * d, seed=3)
        q, k = buffer[:, :H * d].double(), buffer[:, H * d:(H + G) * d].double()
        want_q = plain.rotate_neighbours((plain.rms(q, 1e-5) * wq.double()).reshape(5, H, d), positions, rot).reshape(5, -1)
        want_k = plain.rotate_neighbours((plain.rms(k, 1e-5) * wk.double()).reshape(5, G, d), positions, rot).reshape(5, -1)
        on = buffer.to(DEV)
        freqs = (500.0 ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)).float().to(DEV)
        kernels.wide_norm_rotary(on[:, :H * d], on[:, H * d:(H + G) * d], positions.to(torch.int32).to(DEV), wq.to(DEV), wk.to(DEV), 1e-5,
                                 H, G, d, freqs=freqs, interleaved=True)
        got = on.cpu().double()
        assert (got[:, :H * d] - want_q).abs().max() < 2e-3 and (got[:, H * d:(H + G) * d] - want_k).abs().max() < 2e-3
        assert (got[:3, :H * d] - want_q[:3]).abs().max() < 1e-5


def test_a_stream_changed_between_post_norm_layers_is_rounded_again():
    """The rounded copy of the stream that a post-norm layer hands on is dropped where something else writes the stream: a model
    whose second pass adds a vector, and one with a pre-norm layer between, in bfloat16, against the layers run on fresh
    contexts."""
    from types import SimpleNamespace

    from damendaemon_b200.parts.block import ROUNDED, PostNormBlock
    from damendaemon_b200.parts.interfaces import Runtime
    from damendaemon_b200.parts.norms import RmsNorm
    from damendaemon_b200.parts.spec import NormSpec
    runtime = Runtime(dtype=torch.bfloat16, device=torch.device(DEV))
    norm = RmsNorm(NormSpec("rmsnorm", 32, 1e-5, "w"), {"w": torch.ones(32, device=DEV)}, runtime)
    seen = []

    class Echo:
        def forward_terms(self, y, ctx, cache, position):
            seen.append(y.clone())
            return {"a": y.float()}
    block = PostNormBlock(SimpleNamespace(residual_factor=0.5), [norm], Echo(), None)
    ctx = SimpleNamespace(shared={})
    x = rnd(3, 32, seed=1).to(DEV)
    block.forward(x, ctx, None, None)
    assert torch.equal(ctx.shared[ROUNDED][1], x.to(torch.bfloat16)) and torch.equal(seen[0], rnd(3, 32, seed=1).to(DEV).to(torch.bfloat16))
    block.forward(x, ctx, None, None)
    other = x.clone()
    block.forward(other, ctx, None, None)                # another tensor: its own values are read
    assert torch.equal(seen[2], x.to(torch.bfloat16)) and ctx.shared[ROUNDED][0] is other

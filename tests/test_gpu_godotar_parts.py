"""Each mechanism of Godotar alone: the kernel or part against the plain function of the same name."""
import math

import pytest
import torch

import plain_godotar as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def rnd(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g) * scale


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def layout(lengths):
    """(entry_start, token_entry) of entries of these lengths laid side by side."""
    starts, entry = [0], []
    for e, n in enumerate(lengths):
        starts.append(starts[-1] + n)
        entry += [e] * n
    return starts, entry


# ------------------------------------------------------------------ norms of one row, blends with the token before

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 99, 100, 1600, 3000, 4100])
def test_two_norms_of_one_row(width, dtype):
    from damendaemon_b200 import kernels
    x, w1, w2 = rnd(9, width, seed=1, scale=3.0), rnd(width, seed=2, scale=0.2), rnd(width, seed=3, scale=0.2)
    x[3] *= 1e-3                                            # a row so small that eps matters
    y, z, none = kernels.token_mix(x.to(DEV), w1.to(DEV), 1e-5, dtype, offset=1.0, weight2=w2.to(DEV))
    assert none is None
    tol = 1e-5 if dtype == torch.float32 else 0.03
    assert (y.cpu().double() - plain.norm(x.double(), w1.double(), 1e-5)).abs().max() < tol
    assert (z.cpu().double() - plain.norm(x.double(), w2.double(), 1e-5)).abs().max() < tol


@pytest.mark.parametrize("width,count", [(64, 5), (48, 3), (99, 5), (1024, 5), (1600, 5), (3000, 2), (4100, 5)])
def test_blends_with_the_token_before_over_steps_and_slots(width, count):
    """Three requests in shuffled slots, run in steps of unequal portions (one request left out of a step, portions of one
    and two tokens): every blend equals the plain one over the whole sequence, so the state carried the last normed row; the
    rows have the same bits however the sequence was cut, and the second norm's rows come along."""
    from damendaemon_b200 import kernels
    total, slots = [37, 12, 25], [3, 0, 2]
    xs = [rnd(n, width, seed=40 + i, scale=2.0) for i, n in enumerate(total)]
    w, w2, mu = rnd(width, seed=3, scale=0.2), rnd(width, seed=5, scale=0.2), torch.rand(count, width, generator=torch.Generator().manual_seed(4))
    mu[0, 0], mu[1, 1] = 0.0, 1.0
    normed = [plain.norm(x.double(), w.double(), 1e-5) for x in xs]
    want = [torch.stack([plain.mix(n, mu[s].double()) for s in range(count)]) for n in normed]

    def run(steps, dtype=torch.float32, pad=0):
        state = torch.full((5, width), float("nan"), device=DEV)
        for s in slots:
            state[s].zero_()
        at, rows = [0, 0, 0], [[], [], []]
        for lengths in steps:
            live = [i for i, n in enumerate(lengths) if n]
            x = torch.cat([xs[i][at[i]:at[i] + lengths[i]] for i in live])
            starts, entry = layout([lengths[i] for i in live])
            n = x.shape[0]
            _, z, out = kernels.token_mix(x.to(DEV), w.to(DEV), 1e-5, dtype, offset=1.0, keep=False, weight2=w2.to(DEV), mu=mu.to(DEV),
                                          state=state, token_entry=i32(entry), entry_start=i32(starts),
                                          entry_slot=i32([slots[i] for i in live]), rows_per_mix=n + pad)
            assert (z.cpu().double() - plain.norm(x.double(), w2.double(), 1e-5)).abs().max() < (1e-5 if dtype == torch.float32 else 0.05)
            assert out.shape == (count, n + pad, width)
            for j, i in enumerate(live):
                rows[i].append(out[:, starts[j]:starts[j + 1]].cpu())
                at[i] += lengths[i]
        assert at == total and torch.isnan(state[1]).all() and torch.isnan(state[4]).all()
        for i, s in enumerate(slots):
            assert (state[s].cpu().double() - normed[i][-1]).abs().max() < 1e-5
        return [torch.cat(r, dim=1) for r in rows]
    cut = run([[5, 1, 2], [1, 0, 1], [2, 2, 0], [16, 8, 20], [13, 1, 2]], pad=3)
    whole = run([total])
    for got, other, ref in zip(cut, whole, want):
        assert (got.double() - ref).abs().max() < 1e-5
        assert torch.equal(got, other)
    for got, ref in zip(run([total], dtype=torch.bfloat16, pad=8), want):
        assert (got.double() - ref).abs().max() < 0.05


def test_blends_of_many_tokens_walked_four_to_a_block():
    """2,500 tokens of unequal requests in one step: blocks that walk several tokens meet the borders between requests at every
    place, and the bits are those of small steps."""
    from damendaemon_b200 import kernels
    width, lengths = 64, [1, 2, 3, 1, 700, 1, 1, 90, 1700, 1]
    x, w, mu = rnd(sum(lengths), width, seed=1), rnd(width, seed=2, scale=0.2), torch.rand(5, width, generator=torch.Generator().manual_seed(3))
    starts, entry = layout(lengths)
    kept = rnd(len(lengths), width, seed=4)                       # what earlier steps left
    state = kept.to(DEV)
    _, _, out = kernels.token_mix(x.to(DEV), w.to(DEV), 1e-5, torch.float32, offset=1.0, keep=False, mu=mu.to(DEV), state=state,
                                  token_entry=i32(entry), entry_start=i32(starts), entry_slot=i32(list(range(len(lengths)))))
    for e, n in enumerate(lengths):
        rows = x[starts[e]:starts[e + 1]]
        one = kept[e:e + 1].to(DEV).clone()
        _, _, alone = kernels.token_mix(rows.to(DEV), w.to(DEV), 1e-5, torch.float32, offset=1.0, keep=False, mu=mu.to(DEV), state=one,
                                        token_entry=i32([0] * n), entry_start=i32([0, n]), entry_slot=i32([0]))
        assert torch.equal(out[:, starts[e]:starts[e + 1]], alone) and torch.equal(one[0], state[e]), e
        normed = plain.norm(rows.double(), w.double(), 1e-5)
        before = torch.cat([kept[e:e + 1].double(), normed[:-1]])
        want = torch.stack([normed + (before - normed) * mu[s].double() for s in range(5)])
        assert (alone.cpu().double() - want).abs().max() < 1e-5, e


# ------------------------------------------------------------------ the recurrence

def operands(n, H, dk, dv, seed, slow=-2.0):
    """r, k, v, what enters the decay before its bias, the bias and the bonus; the plain decay."""
    r, k, v = rnd(n, H * dk, seed=seed), rnd(n, H * dk, seed=seed + 1), rnd(n, H * dv, seed=seed + 2)
    x = rnd(n, H * dk, seed=seed + 3)
    return r, k, v, x


def plain_recurrence(ops, w0, u, H, dk, dv):
    r, k, v, x = (t.double() for t in ops)
    n = r.shape[0]
    fade = torch.exp(-torch.exp(x + w0.double()))
    return plain.recurrence(r.view(n, H, dk), k.view(n, H, dk), v.view(n, H, dv), fade.view(n, H, dk), u.double().view(H, dk)).reshape(n, H * dv)


def device_operands(ops, lo, hi, dtype=torch.float32, gate=None):
    """Row views of one buffer, as the projections leave them, and the decay's input."""
    r, k, v, x = (t[lo:hi] for t in ops)
    parts = [r, k, v] + ([gate[lo:hi]] if gate is not None else [])
    buf = torch.cat(parts + [torch.full((r.shape[0], 3), float("nan"))], dim=1).to(dtype).to(DEV)
    views, at = [], 0
    for p in parts:
        views.append(buf[:, at:at + p.shape[1]])
        at += p.shape[1]
    return views, x.contiguous().to(DEV)


def scan(ops, pieces, w0, u, slots, state, H, dk, dv):
    """One step: pieces = [(request, lo, hi)]; ops: a request's operands. Returns each piece's rows."""
    from damendaemon_b200 import kernels
    joined = tuple(torch.cat([ops[i][j][lo:hi] for i, lo, hi in pieces]) for j in range(4))
    starts, _ = layout([hi - lo for _, lo, hi in pieces])
    views, x = device_operands(joined, 0, starts[-1])
    prepared = kernels.time_prepare(*views, x, w0.to(DEV), u.to(DEV), H, dk, dv)
    out = kernels.time_scan(*prepared, i32(starts), i32([slots[i] for i, _, _ in pieces]), state, H, dk, dv).cpu()
    return [out[starts[j]:starts[j + 1]] for j in range(len(pieces))]


@pytest.mark.parametrize("H,dk,dv", [(3, 16, 16), (2, 20, 12), (4, 64, 64), (1, 128, 64), (1, 256, 40), (2, 1, 1), (2, 8, 130), (2, 7, 9), (3, 32, 32)])
def test_the_recurrence_in_portions_with_shuffled_slots(H, dk, dv):
    """Four requests of unequal length in shuffled slots: portions down to two tokens and single tokens, a request left out of a
    step; every output equals the plain recurrence over the whole sequence and has the bits of the whole prompt in one step."""
    from damendaemon_b200 import kernels
    total, slots = [60, 9, 40, 58], [4, 0, 5, 2]
    w0, u = rnd(H * dk, seed=7, scale=1.5) - 2.0, rnd(H * dk, seed=8)
    ops = [operands(n, H, dk, dv, 100 * i) for i, n in enumerate(total)]
    want = [plain_recurrence(o, w0, u, H, dk, dv) for o in ops]

    def run(steps):
        state = torch.full((6, *kernels.delta_state_shape(H, dk, dv)), float("nan"), device=DEV)
        for s in slots:
            state[s].zero_()
        at, rows = [0] * 4, [[] for _ in total]
        for lengths in steps:
            pieces = [(i, at[i], at[i] + n) for i, n in enumerate(lengths) if n]
            for (i, lo, hi), out in zip(pieces, scan(ops, pieces, w0, u, slots, state, H, dk, dv)):
                rows[i].append(out)
                at[i] = hi
        assert at == total and torch.isnan(state[1]).all() and torch.isnan(state[3]).all()
        return [torch.cat(r) for r in rows]
    cut = run([[17, 3, 1, 2], [16, 0, 2, 1], [1, 2, 15, 33], [2, 2, 16, 0], [24, 2, 6, 22]])
    whole = run([total])
    for got, other, ref in zip(cut, whole, want):
        assert (got.double() - ref).abs().max() < 2e-5 * max(1.0, ref.abs().max().item())
        assert torch.equal(got, other)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d", [(3, 16), (2, 20), (2, 64), (1, 128), (1, 256), (5, 1), (2, 40)])
def test_single_tokens_in_one_kernel(H, d, dtype):
    """Two requests decoded side by side for 40 tokens from a prompt's state: operands, recurrence, norm, weight and gate of the
    read-out in one kernel, against the plain functions and against the three kernels of a step with portions."""
    from damendaemon_b200 import kernels
    n, eps, slots = 60, 1e-5, [2, 0]
    w0, u, weight = rnd(H * d, seed=7, scale=1.5) - 2.0, rnd(H * d, seed=8), 1.0 + rnd(H * d, seed=9, scale=0.2)
    ops = [tuple(t.to(dtype).float() if j < 3 else t for j, t in enumerate(operands(n, H, d, d, 50 * i))) for i in range(2)]
    gates = [rnd(n, H * d, seed=70 + i).to(dtype).float() for i in range(2)]
    want = []
    for o, g in zip(ops, gates):
        read = plain_recurrence(o, w0, u, H, d, d)
        want.append(plain.rms(read.view(n, H, d), eps).reshape(n, H * d) * weight.double() * plain.silu(g.double()))
    state = torch.full((3, *kernels.delta_state_shape(H, d, d)), float("nan"), device=DEV)
    state[0].zero_(), state[2].zero_()
    scan(ops, [(0, 0, 20), (1, 0, 20)], w0, u, slots, state, H, d, d)
    other = state.clone()
    for t in range(20, n):
        joined = tuple(torch.stack([ops[0][j][t], ops[1][j][t]]) for j in range(4))
        gate = torch.stack([gates[0][t], gates[1][t]])
        (r, k, v, g), x = device_operands(joined, 0, 2, dtype, gate)
        out = kernels.time_step(r, k, v, g, x, w0.to(DEV), u.to(DEV), weight.to(DEV), eps, i32(slots), state, H, d, d)
        prepared = kernels.time_prepare(r, k, v, x, w0.to(DEV), u.to(DEV), H, d, d)
        read = kernels.time_scan(*prepared, i32([0, 1, 2]), i32(slots), other, H, d, d)
        three = kernels.retention_finish(read, g, H, eps, dtype, weight=weight.to(DEV))
        assert torch.equal(state[0], other[0]) and torch.equal(state[2], other[2]), t
        for i in range(2):
            scale = max(1.0, want[i][t].abs().max().item())
            assert (out[i].cpu().double() - want[i][t]).abs().max() < (5e-5 if dtype == torch.float32 else 0.02) * scale, (t, i)
        assert (out.float() - three.float()).abs().max() < (1e-5 if dtype == torch.float32 else 0.04) * scale, t
    assert torch.isnan(state[1]).all()


def test_a_token_far_back_reaches_the_read_out_through_slow_channels():
    """3,000 tokens without a key behind one marked token, through channels whose decays differ from one by 1e-5 and 4e-6: what is
    left of it is what the plain recurrence leaves, but for the rounding of a float32 state (half an ulp a step, on one side
    for long while nothing is added: at most 1e-4 of the state here)."""
    from damendaemon_b200 import kernels
    H, d, n = 1, 16, 3001
    loss = torch.full((d,), 1e-5, dtype=torch.float64)
    loss[::2] = 4e-6
    w0 = torch.log(loss).float()
    r, k, v, x = (torch.zeros(n, d) for _ in range(4))
    k[0], v[0], r[-1] = rnd(d, seed=1), rnd(d, seed=2), rnd(d, seed=3)
    u = torch.zeros(d)
    want = plain_recurrence((r, k, v, x), w0, u, H, d, d)[-1]
    for cuts in ((0, n), (0, 1, 700, 702, n - 1, n)):
        state = torch.zeros(1, *kernels.delta_state_shape(H, d, d), device=DEV)
        for lo, hi in zip(cuts, cuts[1:]):
            out = scan([(r, k, v, x)], [(0, lo, hi)], w0, u, [0], state, H, d, d)[0]
        assert (out[-1].double() - want).abs().max() < 2e-4 * want.abs().max(), cuts
    # with keys on the way the roundings fall on both sides, and the decay itself is what is left to be wrong
    ops = operands(n, H, d, d, 9)
    want = plain_recurrence((*ops[:3], x), w0, u, H, d, d)
    state = torch.zeros(1, *kernels.delta_state_shape(H, d, d), device=DEV)
    out = scan([(*ops[:3], x)], [(0, 0, n)], w0, u, [0], state, H, d, d)[0]
    assert (out[-500:].double() - want[-500:]).abs().max() < 1e-5 * want[-500:].abs().max()


def test_the_bonus_counts_for_the_current_token_only():
    from damendaemon_b200 import kernels
    H, d = 2, 8
    ops = operands(2, H, d, d, 3)
    w0, big = torch.zeros(H * d), torch.full((H * d,), 1000.0)
    outs = []
    for u in (torch.zeros(H * d), big):
        state = torch.zeros(1, *kernels.delta_state_shape(H, d, d), device=DEV)
        first = scan([ops], [(0, 0, 1)], w0, u, [0], state, H, d, d)[0]
        assert (first.double() - plain_recurrence(ops, w0, u, H, d, d)[:1]).abs().max() < 1e-3
        # the second token is given no key: all it reads is what the first one wrote, whatever its bonus was
        quiet = (ops[0], torch.zeros_like(ops[1]), ops[2], ops[3])
        outs.append(scan([quiet], [(0, 1, 2)], w0, u, [0], state, H, d, d)[0])
    assert torch.equal(outs[0], outs[1]) and outs[0].abs().max() > 0.1


# ------------------------------------------------------------------ latent attention with a query latent, a window and a gate

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,dr,dv,R,Rq,dims,window", [(3, 12, 8, 10, 24, 20, 8, 20), (4, 64, 32, 64, 96, 64, 32, 50), (6, 10, 6, 12, 22, 30, 4, 33),
                                                         (17, 16, 16, 16, 64, 48, 16, None), (40, 8, 24, 8, 136, 32, 24, 64), (1, 8, 2, 8, 14, 12, 2, 1),
                                                         (2, 16, 64, 32, 256, 40, 64, 100)])
def test_the_latent_mixer_against_the_plain_one(H, d, dr, dv, R, Rq, dims, window, dtype):
    """The part itself on a small cache: a prompt of 130 in portions of 77, 2 and 51 rows and 25 single tokens, pages shuffled; its
    output projection is added to the stream."""
    from damendaemon_b200.cache.manager import LayerCache
    from damendaemon_b200.engine.context import StepContext
    from damendaemon_b200.parts import LatentAttentionSpec, Runtime
    from damendaemon_b200.parts.latent_attention import LatentAttention
    from damendaemon_b200.parts.spec import RotarySpec
    from damendaemon_b200 import kernels
    width, T, P, eps, base = 64, 155, 16, 1e-5, 300.0
    t = getattr(torch, dtype)
    shapes = {"dq": (Rq, width), "uq": (H * (d + dr), Rq), "dkv": (R + dr, width), "uk": (H * d, R), "uv": (H * dv, R), "g": (H, width),
              "o": (width, H * dv)}
    w = {n: (rnd(*s, seed=i) / math.sqrt(s[1])).to(t) for i, (n, s) in enumerate(shapes.items())}
    w["dq.norm"], w["dkv.norm"] = 2.0 + rnd(Rq, seed=20, scale=0.2), 1.0 + rnd(R, seed=21, scale=0.2)
    h = rnd(T, width, seed=22).to(t)
    m = {"heads": H, "dim": d, "rot_dim": dr, "vdim": dv, "kv_rank": R, "q_rank": Rq, "scale": (d + dr) ** -0.5, "rot": {"dims": dims, "base": base}}
    if window:
        m["mask"] = {"size": window}
    want = plain.latent_attention(h.double(), {"m." + n: v.double() for n, v in w.items()}, "m.", m, eps)
    spec = LatentAttentionSpec("latent_attention", width=width, n_heads=H, head_dim=d, rot_dim=dr, value_dim=dv, rank=R, scale=m["scale"],
                               norm_eps=eps, rotary=RotarySpec("rotary", dr, dims, base, interleaved=False), query_weight="uq",
                               down_weight="dkv", latent_norm="dkv.norm", up_key_weight="uk", up_value_weight="uv", out_weight="o",
                               window=window, gate_weight="g", query_down="dq", query_norm="dq.norm", query_rank=Rq)
    placed = {}
    for decl in LatentAttention.tensor_decls(spec):
        placed[decl.name] = (torch.cat([w[n] for n, _ in decl.pieces]) if decl.pieces else w[decl.name]).to(DEV)
    runtime = Runtime(dtype=t, device=torch.device(DEV))
    part = LatentAttention(spec, placed, runtime)
    need, = LatentAttention.cache_needs(spec)
    assert need.window == window and need.width == R + dr

    class Group:
        name = "rows"
    n_pages = 13
    order = torch.randperm(n_pages, generator=torch.Generator().manual_seed(6))[:-(-T // P)].tolist()
    cache = LayerCache(Group, torch.full((n_pages, P * (R + dr)), float("nan"), dtype=t, device=DEV), None, P)
    got = []
    cuts = [0, 77, 79, 130] + list(range(131, T + 1))
    for lo, hi in zip(cuts, cuts[1:]):
        n = hi - lo
        table = list(order) + [-1]
        if window:                                   # pages that the window has passed may belong to somebody else by now
            for b in range(max(0, lo - window + 1) // P):
                table[b] = -1
        ctx = StepContext(n_tokens=n, n_entries=1, n_wanted=0, token_ids=None, positions=i32(list(range(lo, hi))), token_entry=i32([0] * n),
                          want_rows=None, entry_slot=i32([0]), entry_start=i32([0, n]), entry_pos0=i32([lo]), block_tables={"rows": i32([table])},
                          decode_only=n == 1, split_context=hi, runtime=runtime)
        stream = rnd(n, width, seed=lo)
        out = part.forward(h[lo:hi].to(DEV), stream.to(DEV), ctx, cache, None)
        got.append(out.cpu().double() - stream.double())
    assert kernels.read_error_flag(DEV) == 0
    err = (torch.cat(got) - want).abs().max().item()
    assert err < (5e-5 if dtype == "float32" else 0.06) * max(1.0, want.abs().max().item()), err


@pytest.mark.parametrize("kernel", ["tensor", "rows"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [1, 7, 16, 33, 64, 65, 200])
def test_a_marked_latent_row_at_the_windows_edges(window, decode, kernel):
    """600 rows of noise and one whose last element answers the query a hundred times better: seen from its own place up to
    window - 1 places later, and neither before nor after, at page and tile borders, in a prompt and alone with key splits;
    a gate of sigmoid(1) multiplies what is seen."""
    from damendaemon_b200 import kernels
    H, R, dr, P, T = 3, 32, 16, 16, 600
    row, gate_value = R + dr, 1.0 / (1.0 + math.exp(-1.0))
    gate = torch.ones(T, H, dtype=torch.bfloat16, device=DEV)
    for marked in (0, 63, 64, 16 * 17 - 1, 300):
        rows = (rnd(T, row, seed=marked + 1) * 0.05).to(torch.bfloat16)
        rows[marked, :R] = torch.arange(R) / 8.0 - 2.0
        rows[marked, row - 1] = 6.0
        cache = torch.cat([rows.view(-1), torch.zeros((-T % P) * row, dtype=torch.bfloat16)]).view(-1, P * row).to(DEV)
        q = torch.zeros(T, H * row, dtype=torch.bfloat16)
        q.view(T, H, row)[:, :, row - 1] = 6.0
        q = q.to(DEV)
        places = [p for p in (marked - 1, marked, marked + window - 1, marked + window) if 0 <= p < T]
        lo = max(0, min(places) - 5)
        hi = max(places) + 1
        table = list(range(cache.shape[0]))
        for b in range(max(0, (lo if not decode else 0) - window + 1) // P):
            table[b] = -1                              # given back
        for at in places:
            if decode:
                mine = [(-1 if b < max(0, at - window + 1) // P else b) for b in range(cache.shape[0])]
                if kernel == "tensor":
                    out = kernels.attention_latent(q[at:at + 1], cache, i32([0, 1]), i32([at]), i32([mine]), H, R, 1.0, n_splits=3, window=window,
                                                   gate=gate[:1])[0]
                else:
                    out = kernels.attention_rows(q[at:at + 1], cache, i32([0]), i32([at]), i32([mine]), H, 1.0, window=window, n_splits=3,
                                                 kv_heads=1, v_dim=R, values_in_keys=True, gate=gate[:1])[0]
            elif kernel == "tensor":
                out = kernels.attention_latent(q[lo:hi], cache, i32([0, hi - lo]), i32([lo]), i32([table]), H, R, 1.0, window=window,
                                               gate=gate[lo:hi])[at - lo]
            else:
                out = kernels.attention_rows(q[lo:hi], cache, i32([0] * (hi - lo)), i32(list(range(lo, hi))), i32([table]), H, 1.0, window=window,
                                             kv_heads=1, v_dim=R, values_in_keys=True, gate=gate[lo:hi])[at - lo]
            out = out.float().cpu().view(H, R)
            if marked <= at < marked + window:
                assert (out - rows[marked, :R].float() * gate_value).abs().max() < 0.02, (marked, at)
            else:
                assert out.abs().max() < 0.2, (marked, at)
    assert kernels.read_error_flag(DEV) == 0


def test_a_far_latent_row_among_hundreds_is_found_without_a_window():
    from damendaemon_b200 import kernels
    H, R, dr, P, T = 2, 64, 32, 16, 1500
    row = R + dr
    for marked in (5, 640, 1023, 1024):
        rows = (rnd(T, row, seed=marked) * 0.05).to(torch.bfloat16)
        rows[marked, row - 1] = 6.0
        cache = torch.cat([rows.view(-1), torch.zeros((-T % P) * row, dtype=torch.bfloat16)]).view(-1, P * row).to(DEV)
        q = torch.zeros(1, H * row, dtype=torch.bfloat16)
        q.view(H, row)[:, row - 1] = 6.0
        out = kernels.attention_latent(q.to(DEV), cache, i32([0, 1]), i32([T - 1]), i32([list(range(cache.shape[0]))]), H, R, 1.0, n_splits=7)
        assert (out.float().cpu().view(H, R) - rows[marked, :R].float()).abs().max() < 0.02


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("interleaved", [False, True])
def test_latent_rows_with_a_second_latent_and_turned_tails(interleaved, dtype):
    """The prepare kernel without queries: the cache row and the normed second latent; and the queries' rotated parts turned
    while the per-head product (both kernels) carries them, at positions up to 5,000."""
    from damendaemon_b200 import kernels
    n, H, d, dr, R, S, dims, P, base, eps = 70, 3, 16, 24, 40, 56, 16, 16, 200.0, 1e-5
    pos = torch.arange(n) + 4930
    proj = rnd(n, S + R + dr + 3, seed=1).to(dtype)
    wl, ws = 1.0 + rnd(R, seed=2, scale=0.2), 1.0 + rnd(S, seed=3, scale=0.2)
    freqs = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    rot = {"dims": dims, "base": base}

    def turned(x):                                      # [n, heads, dr]
        if not interleaved:
            return plain.rotate_halves(x, pos, rot)
        a, b = x[..., 0:dims:2], x[..., 1:dims:2]
        angle = pos.double()[:, None] * freqs[None]
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        both = torch.stack([a * c - b * s, b * c + a * s], dim=-1).flatten(-2)
        return torch.cat([both, x[..., dims:]], dim=-1)
    pages = -(-5000 // P)
    cache = torch.zeros((pages, P * (R + dr)), dtype=dtype, device=DEV)
    dev = proj.to(DEV)
    second = kernels.latent_prepare(None, dev[:, S:S + R + dr], wl.to(DEV), eps, freqs.float().to(DEV), i32([0] * n), i32(pos.tolist()),
                                    i32([list(range(pages))]), cache, H, d, dr, R, interleaved=interleaved, second=dev[:, :S], second_weight=ws.to(DEV))
    tol = 3e-3 if dtype == torch.float32 else 0.04         # (angles of thousands of radians are float32)
    want = plain.rms(proj[:, :S].double(), eps) * ws.double()
    assert (second.cpu().double() - want).abs().max() < (1e-5 if dtype == torch.float32 else 0.03)
    down = proj[:, S:S + R + dr].double()
    want = torch.cat([plain.rms(down[:, :R], eps) * wl.double(), turned(down[:, None, R:])[:, 0]], dim=1)
    got = cache.cpu().double().view(-1, R + dr)[pos]
    assert (got - want).abs().max() < tol
    q = rnd(n, H * (d + dr), seed=5).to(dtype)
    w = (rnd(H, R, d, seed=6) / math.sqrt(d)).to(dtype)
    heads = q.double().view(n, H, d + dr)
    want = torch.cat([torch.einsum("nhi,hji->nhj", heads[..., :d], w.double()), turned(heads[..., d:])], dim=-1)
    for kernel in ("plain", "mma") if dtype == torch.bfloat16 else ("plain",):
        got = kernels.per_head_linear(q.to(DEV), w.to(DEV), d + dr, tail=dr, kernel=kernel, turn=(freqs.float().to(DEV), i32(pos.tolist()), interleaved))
        assert (got.cpu().double().view(n, H, R + dr) - want).abs().max() < tol, kernel
    assert kernels.read_error_flag(DEV) == 0


# ------------------------------------------------------------------ experts by a softmax router

@pytest.mark.parametrize("dtype,width", [(torch.float32, 64), (torch.bfloat16, 256), (torch.float32, 99)])
@pytest.mark.parametrize("outputs,top", [(10, 2), (5, 1), (6, 6), (64, 7), (33, 3), (2, 1)])
def test_the_softmax_router_with_a_correction(outputs, top, dtype, width):
    from damendaemon_b200 import kernels
    tokens = 300
    y = rnd(tokens, width, seed=outputs + top).to(dtype)
    router, correction = rnd(outputs, width, seed=outputs, scale=2.0 * width ** -0.5).to(dtype), rnd(outputs, seed=1, scale=0.3)
    z = y.double() @ router.double().T
    for c in (correction, torch.zeros(outputs), correction - 5.0):
        want, weight = plain.choose(z, c.double(), top)
        chosen, got, none = kernels.route_by_score(y.to(DEV), router.to(DEV), outputs, top, softmax=True, correction=c.to(DEV), renormalize=True)
        assert none is None and torch.equal(chosen.cpu().long(), want)
        assert (got.cpu().double() - weight).abs().max() < 3e-6
    scores = torch.softmax(z, dim=-1)
    chosen, got, _ = kernels.route_by_score(y.to(DEV), router.to(DEV), outputs, top, softmax=True, weight_scale=2.0)
    assert (got.cpu().double() - 2.0 * scores.gather(1, chosen.cpu().long())).abs().max() < 6e-6
    # the correction beside sigmoid scores, and logits far apart
    chosen, got, _ = kernels.route_by_score(y.to(DEV), router.to(DEV), outputs, top, correction=correction.to(DEV))
    sig = torch.sigmoid(z)
    want = torch.topk(sig + correction.double(), top, dim=-1).indices
    assert torch.equal(chosen.cpu().long(), want) and (got.cpu().double() - sig.gather(1, want)).abs().max() < 3e-6
    chosen, got, _ = kernels.route_by_score((y * 200).to(DEV), router.to(DEV), outputs, 1, softmax=True, renormalize=True)
    assert torch.equal(chosen.cpu()[:, 0].long(), ((y * 200).double() @ router.double().T).argmax(-1)) and (got == 1.0).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,identity,tokens", [(8, 2, 2, 1), (5, 2, 3, 37), (3, 5, 2, 200), (4, 1, 0, 60), (2, 2, 6, 70), (1, 1, 1, 5), (16, 3, 1, 300)])
def test_experts_and_identity_outputs(experts, top, identity, tokens, dtype):
    from damendaemon_b200.parts import GatedUnitSpec, Runtime, ScoreRoutedExpertsSpec
    from damendaemon_b200.parts.feed_forward import ScoreRoutedExperts
    width, inner, limit = 64, 24, 0.8
    w = {}
    for e in range(experts):
        w[f"e{e}.gate"], w[f"e{e}.up"] = rnd(inner, width, seed=20 + len(w), scale=0.3), rnd(inner, width, seed=21 + len(w), scale=0.3)
        w[f"e{e}.down"] = rnd(width, inner, seed=22 + len(w), scale=0.3)
    w["router"] = rnd(experts + identity, width, seed=3, scale=0.4)
    correction = rnd(experts + identity, seed=4, scale=0.2)
    y, stream = rnd(tokens, width, seed=30), rnd(tokens, width, seed=31)
    f = {"router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": inner, "limit": limit}}
    rounded = {k: t.to(dtype).double() for k, t in w.items()}
    rounded["correction"] = correction.double()
    want = stream.double() + plain.experts(y.to(dtype).double(), rounded, "", f)
    spec = ScoreRoutedExpertsSpec("experts_by_score", width, top, "router",
                                  tuple(GatedUnitSpec(inner, limit, f"e{e}.gate", f"e{e}.up", f"e{e}.down") for e in range(experts)),
                                  score="softmax", correction="correction", renormalize=True, identity=identity)
    assert {d.name for d in ScoreRoutedExperts.tensor_decls(spec)} == set(w) | {"correction"}
    weights = {k: t.to(dtype).to(DEV) for k, t in w.items()}
    weights["correction"] = correction.to(DEV)
    part = ScoreRoutedExperts(spec, weights, Runtime(dtype=dtype, device=torch.device(DEV)))
    got = part.forward(y.to(dtype).to(DEV), stream.clone().to(DEV), None).cpu().double()
    assert (got - want).abs().max() < (5e-6 if dtype == torch.float32 else 0.01) * max(1.0, want.abs().max().item())
    from damendaemon_b200 import kernels
    assert kernels.read_error_flag(DEV) == 0


def test_a_choice_outside_the_outputs_is_an_error():
    from damendaemon_b200 import kernels
    for bad in (7, -2, -1):
        table = i32([[0, 5], [bad, 6]])
        pair_row, _, _ = kernels.route_by_table(None, table, 5, 16, n_identity=2)
        assert kernels.read_error_flag(DEV) == 1
        assert pair_row.cpu().tolist()[1:] == [-2, -1, -2]
    kernels.route_by_table(None, i32([[0, 5], [4, 6]]), 5, 16, n_identity=2)
    assert kernels.read_error_flag(DEV) == 0


# ------------------------------------------------------------------ small pieces

@pytest.mark.parametrize("m,n,k", [(1, 16, 256), (8, 5, 64), (40, 64, 1600), (100, 24, 100), (300, 64, 512), (2048, 16, 64)])
def test_products_with_tanh_in_their_epilogue(m, n, k):
    from damendaemon_b200 import kernels
    a, w = rnd(m, k, seed=1), rnd(n, k, seed=2) / math.sqrt(k)
    got = kernels.gemm_simt(a.to(DEV), w.to(DEV), activation="tanh")
    assert (got.cpu().double() - torch.tanh(a.double() @ w.double().T)).abs().max() < 1e-5
    a, w = a.to(torch.bfloat16), w.to(torch.bfloat16)
    want = torch.tanh(a.double() @ w.double().T)
    if k % 8 == 0:
        assert (kernels.gemm_tcgen05(a.to(DEV), w.to(DEV), activation="tanh").cpu().double() - want).abs().max() < 0.01
        assert (kernels.gemm_tcgen05(a.to(DEV), w.to(DEV), activation="tanh", out_dtype=torch.float32).cpu().double() - want).abs().max() < 1e-4
    assert (kernels.gemm_simt(a.to(DEV), w.to(DEV), activation="tanh", out_dtype=torch.float32).cpu().double() - want).abs().max() < 1e-5


@pytest.mark.parametrize("kind", ["rmsnorm", "layernorm", "tanh"])
def test_a_scale_of_the_logits_is_folded_into_the_heads_norm(kind):
    from damendaemon_b200.parts import Runtime
    from damendaemon_b200.parts.head import LinearHead
    from damendaemon_b200.parts.spec import HeadSpec, NormSpec
    width, vocab = 48, 31
    weights = {"n": rnd(width, seed=1, scale=0.2).to(DEV), "n.b": rnd(width, seed=2, scale=0.2).to(DEV), "n.a": torch.tensor(0.5, device=DEV),
               "w": rnd(vocab, width, seed=3).to(DEV), "b": rnd(vocab, seed=4).to(DEV)}
    norm = NormSpec(kind, width, 1e-5, "n", bias=None if kind == "rmsnorm" else "n.b", alpha="n.a" if kind == "tanh" else None,
                    weight_offset=1.0 if kind == "rmsnorm" else 0.0)

    class Context:
        want_rows = i32([4, 0, 2])
    x = rnd(6, width, seed=5).to(DEV)
    runtime = Runtime(dtype=torch.float32, device=torch.device(DEV))
    for bias in (None, "b"):
        head = lambda scale: LinearHead(HeadSpec("linear", vocab, width, norm, "w", bias=bias, scale=scale), weights, runtime).forward(x, Context)
        assert (head(0.37) - 0.37 * head(1.0)).abs().max() < 1e-5


def test_a_step_of_single_tokens_equals_the_same_rows_as_a_portion():
    """The mixer part: four tokens of one request, one by one, against the same four as one portion, in both dtypes, and a step of
    more tokens than the grouped product takes."""
    from damendaemon_b200 import kernels
    from damendaemon_b200.cache.manager import LayerCache
    from damendaemon_b200.engine.context import StepContext
    from damendaemon_b200.parts import Runtime, TimeMixSpec
    from damendaemon_b200.parts.block import normed_mixer
    from damendaemon_b200.parts.norms import RmsNorm
    from damendaemon_b200.parts.spec import NormSpec
    from damendaemon_b200.parts.time_mix import TimeMix
    width, H, d, rank, T = 96, 3, 24, 8, 150
    spec = TimeMixSpec("time_mix", width, H, d, rank, 1e-5, tuple("mu." + s for s in "rkvgw"), "r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o")
    for dtype in (torch.float32, torch.bfloat16):
        w = {}
        for decl in TimeMix.tensor_decls(spec):
            for name, shape in decl.pieces or ((decl.name, decl.shape),):
                t = rnd(*shape, seed=len(w) + 1)
                w[name] = (t / math.sqrt(shape[-1])).to(dtype) if decl.role == "matrix" else torch.sigmoid(t) if name.startswith("mu.") else t
        placed = {decl.name: (torch.cat([w[n] for n, _ in decl.pieces]) if decl.pieces else w[decl.name]).to(DEV) for decl in TimeMix.tensor_decls(spec)}
        placed["n1"] = torch.zeros(width, device=DEV)
        runtime = Runtime(dtype=dtype, device=torch.device(DEV))
        part = TimeMix(spec, placed, runtime)
        norm = RmsNorm(NormSpec("rmsnorm", width, 1e-5, "n1", weight_offset=1.0), placed, runtime)
        x = rnd(T, width, seed=40)
        h = plain.norm(x.double(), torch.zeros(width, dtype=torch.float64), 1e-5)
        want = plain.time_mixer(h, {"m." + n: t.double() for n, t in w.items()}, "m.", {"heads": H, "dim": d}, 1e-5)
        for cuts in ([0, T], [0, 130, 132] + list(range(133, T + 1)), [0, 100] + list(range(101, T + 1))):
            cache = LayerCache(None, None, torch.zeros(1, *kernels.delta_state_shape(H, d, d), device=DEV), 16,
                               named={"shift": torch.zeros(1, width, device=DEV)})
            got = []
            for lo, hi in zip(cuts, cuts[1:]):
                n = hi - lo
                ctx = StepContext(n_tokens=n, n_entries=1, n_wanted=0, token_ids=None, positions=i32(list(range(lo, hi))), token_entry=i32([0] * n),
                                  want_rows=None, entry_slot=i32([0]), entry_start=i32([0, n]), entry_pos0=i32([lo]), block_tables={},
                                  decode_only=n == 1, runtime=runtime)
                out = normed_mixer(norm, part, x[lo:hi].to(DEV), ctx, cache, None)
                got.append(out.cpu().double() - x[lo:hi].double())
            err = (torch.cat(got) - want).abs().max().item()
            assert err < (5e-5 if dtype == torch.float32 else 0.08) * max(1.0, want.abs().max().item()), (dtype, len(cuts), err)

"""The kernels behind Birelix's mechanisms, each alone against its plain function (`plain_birelix.py`): the short convolutions
and unit vectors, the delta rule (portions and single tokens of several requests through their slots, a value that one write
left and the last query asks for, rewritten keys), a decode step in one kernel, the gate per head, attention with unit queries
and keys, a window and one added to the denominator in every kernel with keys that stand out just inside and just outside the
window, routing by pairs of group scores with renormalised weights, experts with a bounded gate in every grouped product."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_birelix as P

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
TOL = {torch.float32: 2e-5, torch.bfloat16: 8e-3}   # (a bfloat16 result is rounded once: 2^-8 of its size)


def dev(x, dtype=torch.float32):
    return torch.from_numpy(np.array(x, dtype=np.float64, order="C")).to(DEV).to(dtype)


def ints(x):
    return torch.tensor([int(v) for v in x], dtype=torch.int32, device=DEV)


def bf(x):
    return P.store_bfloat16(x)


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def close(got, want, tol):
    got = host(got)
    scale = max(1.0, float(np.abs(want).max()))
    assert got.shape == want.shape and np.isfinite(got).all()
    assert np.abs(got - want).max() <= tol * scale, "largest error %g of scale %g" % (np.abs(got - want).max(), scale)


def step_of(lens, starts, slots):
    """The fields of a step's context that the delta rule's kernels read."""
    cu = np.concatenate([[0], np.cumsum(lens)])
    pos = np.concatenate([np.arange(s, s + n) for s, n in zip(starts, lens)])
    return SimpleNamespace(n_seqs=len(lens), max_new=max(lens), cu_seqlens=ints(cu), state_slots=ints(slots), positions=ints(pos),
                           seq_of_token=ints(np.repeat(np.arange(len(lens)), lens)))


# -- the delta rule ----------------------------------------------------------------------------------------------------------

class Rule:
    """Random inputs of several sequences for one set of sizes, and what the plain functions make of them."""

    def __init__(self, G, H, D, Dv, taps, lens, seed, slow=False):
        rng = np.random.default_rng(seed)
        self.G, self.H, self.D, self.Dv, self.taps, self.lens = G, H, D, Dv, taps, lens
        self.C = 2 * G * D + H * Dv
        self.x = [bf(rng.normal(size=(n, self.C + H * Dv))) for n in lens]          # q, k, v and the gates
        self.ab = [rng.normal(size=(n, 2 * H)) * 2.0 for n in lens]                 # b, then a
        self.w = bf(rng.normal(size=(self.C, taps)) * 0.7)
        self.a_log = rng.uniform(-12.0, -11.0, H) if slow else rng.uniform(-4.0, 1.0, H)
        self.dt = rng.normal(size=H)
        self.norm = 1.0 + 0.2 * rng.normal(size=Dv)

    def args(self):
        return dev(self.w.T), dev(-np.exp(self.a_log)), dev(self.dt)

    def plain(self, i, state=None):
        """(y before the walk, o, the state after it)"""
        G, H, D, Dv, x, ab = self.G, self.H, self.D, self.Dv, self.x[i], self.ab[i]
        T = len(x)
        y = P.short_convolution(x[:, :self.C], self.w)
        q, k = (P.unit_vector(y[:, j * G * D:(j + 1) * G * D].reshape(T, G, D)) for j in (0, 1))
        g = np.exp(-np.exp(self.a_log) * P.softplus(ab[:, H:] + self.dt))
        return P.delta_walk(q * D ** -0.5, k, y[:, 2 * G * D:].reshape(T, H, Dv), g, P.sigmoid(ab[:, :H]), state)

    def finished(self, i, o):
        gate = self.x[i][:, self.C:].reshape(o.shape)
        return (P.rms_norm(o, self.norm, 1e-5) * P.silu(gate)).reshape(len(o), -1)

    def buffers(self, slots=4):
        """State and ring, filled with what no request may read."""
        state = torch.full((slots, self.H, self.Dv, self.D), 7.0, device=DEV)
        ring = torch.full((slots, self.taps, self.C), float("nan"), device=DEV)
        return state, ring

    def run(self, ctx, rows, state, ring, dtype, layout=0):
        from velox_b200.csrc import ops
        x = dev(np.concatenate([self.x[i][a:b] for i, a, b in rows]), dtype)
        ab = dev(np.concatenate([self.ab[i][a:b] for i, a, b in rows]))
        return ops.delta_rule(x, ab, self.H, 0, *self.args(), state, ring, ctx, self.G, self.D, self.H, self.Dv, self.D ** -0.5, layout=layout)

    def decode(self, ctx, rows, state, ring, x_dtype, dtype):
        from velox_b200.csrc import ops
        x = dev(np.concatenate([self.x[i][a:b] for i, a, b in rows]), x_dtype)
        ab = dev(np.concatenate([self.ab[i][a:b] for i, a, b in rows]))
        args = self.args()
        norm = dev(self.norm)
        torch.cuda.synchronize()   # (state and ring have to be older than the kernel before this one)
        out = ops.delta_decode(x, self.C, ab, self.H, 0, *args, norm, state, ring, ctx, self.G, self.D, self.H, self.Dv,
                               self.D ** -0.5, 1e-5, dtype)
        torch.cuda.synchronize()
        return out


SIZES = [(2, 4, 64, 64, 4), (1, 2, 128, 128, 4), (3, 3, 32, 48, 4), (2, 2, 12, 20, 3), (1, 3, 130, 140, 7), (2, 4, 200, 12, 5), (1, 1, 1, 1, 1),
         (1, 2, 256, 33, 2), (2, 6, 36, 8, 4), (4, 4, 64, 30, 4), (1, 1, 7, 300, 9)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("G,H,D,Dv,taps", SIZES)
def test_portions_and_single_tokens_of_several_requests_through_their_slots(dtype, G, H, D, Dv, taps):
    """Three sequences in steps of unequal portions (also one and two tokens, shorter than the convolutions reach back; one left out
    of a step; portions that are no multiple of a mini-chunk or a staged chunk), then single tokens in the one-kernel step."""
    r = Rule(G, H, D, Dv, taps, [63, 29, 80], D + Dv)
    slots, at = [2, 0, 3], [0, 0, 0]
    state, ring = r.buffers()
    for s in slots:
        state[s] = 0.0
    want = [r.plain(i) for i in range(3)]
    for plan in ([5, 1, 2], [1, 1, 1], [0, 2, 33], [16, 5, 0], [1, 0, 4], [33, 17, 36]):
        who = [i for i in range(3) if plan[i]]
        rows = [(i, at[i], at[i] + plan[i]) for i in who]
        ctx = step_of([plan[i] for i in who], [at[i] for i in who], [slots[i] for i in who])
        got = r.run(ctx, rows, state, ring, dtype)
        close(got, np.concatenate([want[i][0][a:b].reshape(b - a, -1) for i, a, b in rows]), 3e-5)
        for i in who:
            at[i] += plan[i]
    for _ in range(3):
        rows = [(i, at[i], at[i] + 1) for i in range(3)]
        got = r.decode(step_of([1, 1, 1], at, slots), rows, state, ring, dtype, dtype)
        close(got, np.concatenate([r.finished(i, want[i][0])[a:b] for i, a, b in rows]), max(TOL[dtype], 5e-5))
        at = [a + 1 for a in at]
    rest = [n - a for n, a in zip(r.lens, at)]
    who = [i for i in range(3) if rest[i]]
    got = r.run(step_of([rest[i] for i in who], [at[i] for i in who], [slots[i] for i in who]), [(i, at[i], r.lens[i]) for i in who], state, ring, dtype)
    close(got, np.concatenate([want[i][0][at[i]:].reshape(rest[i], -1) for i in who]), 3e-5)
    for i in range(3):
        close(state[slots[i]].transpose(1, 2), want[i][1], 3e-5)
        n = r.lens[i]
        for p in range(max(0, n - taps + 1), n):
            close(ring[slots[i], p % taps], r.x[i][p, :r.C], 0.0)
    assert (state[1] == 7.0).all() and torch.isnan(ring[1]).all()


@pytest.mark.parametrize("G,H,D,Dv,taps", [(2, 4, 64, 64, 4), (1, 1, 128, 128, 4), (2, 2, 12, 20, 3), (1, 2, 256, 16, 4)])
def test_how_a_sequence_is_cut_changes_nothing_but_rounding(G, H, D, Dv, taps):
    r = Rule(G, H, D, Dv, taps, [150], 5)
    want = r.plain(0)[0].reshape(150, -1)
    for sizes in ([150], [2], [1, 16, 3], [64, 86], [147, 3]):
        state, ring = r.buffers()
        state[1] = 0.0
        at, k = 0, 0
        while at < 150:
            n = min(sizes[k % len(sizes)], 150 - at)
            got = r.run(step_of([n], [at], [1]), [(0, at, at + n)], state, ring, torch.float32)
            close(got, want[at:at + n], 2e-5)
            at, k = at + n, k + 1


@pytest.mark.parametrize("G,H,D,Dv,taps", [(2, 4, 64, 64, 4), (1, 2, 128, 40, 4), (2, 2, 12, 20, 3), (1, 2, 256, 33, 4)])
def test_columns_a_warp_holds_change_no_bit_and_many_requests_take_more(G, H, D, Dv, taps):
    """Both layouts of the walk, and the one the kernel chooses: two requests, then forty (more blocks than the GPU has places for
    at once), each with the bits it has alone."""
    lens = [37, 16] + [3 + i for i in range(38)]
    r = Rule(G, H, D, Dv, taps, lens, 6)
    outs = []
    for layout in (1, 2, 0):
        state, ring = r.buffers(40)
        state[:] = 0.0
        outs.append(r.run(step_of(lens[:2], [0, 0], [1, 0]), [(0, 0, 37), (1, 0, 16)], state, ring, torch.float32, layout))
    assert torch.equal(outs[0], outs[1]) and torch.equal(outs[0], outs[2])
    close(outs[0][:37], r.plain(0)[0].reshape(37, -1), 2e-5)
    for layout in (1, 2, 0):
        state, ring = r.buffers(40)
        state[:] = 0.0
        many = r.run(step_of(lens, [0] * 40, range(40)), [(i, 0, n) for i, n in enumerate(lens)], state, ring, torch.float32, layout)
        assert torch.equal(many[:53], outs[0])
        close(many[-lens[-1]:], r.plain(39)[0].reshape(lens[-1], -1), 2e-5)


@pytest.mark.parametrize("D,Dv,T", [(64, 64, 700), (128, 32, 300), (20, 12, 700)])
@pytest.mark.parametrize("single", [False, True])
def test_a_value_written_long_ago_is_found_and_a_rewritten_one_is_not(D, Dv, T, single):
    """No decay to speak of and one tap: the first token's value lies under a key that no other key touches until the last query asks
    for it; a second key is written twice, and a query for it finds the second value alone."""
    rng = np.random.default_rng(T)
    r = Rule(1, 1, D, Dv, 1, [T], 3, slow=True)
    r.w[:] = 1.0
    x = r.x[0]
    x[:, :2 * D] = np.abs(x[:, :2 * D])
    x[:, D:D + 2], x[:, :D] = -40.0, -40.0                      # (silu of -40 is nothing: keys and queries without the first two channels)
    x[:, 2] = 3.0
    for t, c in ((0, 0), (1, 1), (T // 2, 1)):                   # three writes, to channel 0 and, twice, to channel 1
        x[t, D:2 * D], x[t, D + c] = -40.0, 5.0
    for t, c in ((T - 1, 0), (T - 2, 1)):
        x[t, :D], x[t, c] = -40.0, 5.0
    r.ab[0][:, 0] = 30.0                                         # steps of one
    x[:] = bf(x)
    want, _ = r.plain(0)
    v = P.silu(x[:, 2 * D:2 * D + Dv])
    s = D ** -0.5
    assert np.abs(want[T - 1, 0] - s * v[0]).max() < 0.02 and np.abs(want[T - 2, 0] - s * v[T // 2]).max() < 0.02
    state, ring = r.buffers()
    state[0] = 0.0
    if not single:
        got = r.run(step_of([T], [0], [0]), [(0, 0, T)], state, ring, torch.float32)
        close(got, want.reshape(T, -1), 2e-5)
        return
    r.run(step_of([T - 8], [0], [0]), [(0, 0, T - 8)], state, ring, torch.float32)
    done = r.finished(0, want)
    for t in range(T - 8, T):
        close(r.decode(step_of([1], [t], [0]), [(0, t, t + 1)], state, ring, torch.float32, torch.float32), done[t:t + 1], 1e-4)


@pytest.mark.parametrize("x_dtype,dtype", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("G,H,D,Dv,taps", SIZES)
def test_a_step_of_single_tokens_from_the_first_position(x_dtype, dtype, G, H, D, Dv, taps):
    """Twelve steps of two requests that start together, beside a third that comes two steps later: before position taps - 1 the
    convolutions reach before the start, whatever the ring holds."""
    r = Rule(G, H, D, Dv, taps, [12, 12, 10], 40 + D)
    state, ring = r.buffers()
    for s in (1, 3, 0):
        state[s] = 0.0
    done = [r.finished(i, r.plain(i)[0]) for i in range(3)]
    for t in range(12):
        who = [(0, t, 1), (1, t, 3)] + ([(2, t - 2, 0)] if t >= 2 else [])
        rows = [(i, p, p + 1) for i, p, _ in who]
        got = r.decode(step_of([1] * len(who), [p for _, p, _ in who], [s for *_, s in who]), rows, state, ring, x_dtype, dtype)
        close(got, np.concatenate([done[i][a:b] for i, a, b in rows]), max(TOL[dtype], 5e-5))
    assert (state[2] == 7.0).all() and torch.isnan(ring[2]).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,V", [(1, 1, 1), (5, 3, 14), (70, 4, 64), (9, 2, 33), (300, 16, 128)])
def test_the_gate_per_head(dtype, T, H, V):
    from velox_b200.csrc import ops
    rng = np.random.default_rng(V)
    o, wide = bf(rng.normal(size=(T, H * V))), bf(rng.normal(size=(T, H + 5)) * 2.0)
    want = (o.reshape(T, H, V) * P.sigmoid(wide[:, 2:2 + H])[:, :, None]).reshape(T, -1)
    close(ops.head_gate(dev(o, dtype), dev(wide, dtype)[:, 2:2 + H]), want, TOL[dtype])


# -- attention -----------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv,window", [(4, 2, 10, 12, 7), (4, 2, 64, 64, 40), (2, 1, 128, 64, 16), (4, 1, 128, 128, 100), (6, 2, 32, 32, 33),
                                             (2, 2, 64, 32, 1), (3, 1, 21, 21, 130)])
def test_unit_queries_and_keys_in_every_kernel_where_keys_stand_out_at_the_windows_edge(dtype, H, G, D, Dv, window):
    """Biased projections whose queries and keys are divided by their root mean square and written to scattered pages; then, in every
    kernel that takes the sizes: query t has one key of its own making exactly window - 1 tokens before it (which it must see) and the
    same one window tokens before it (which it must not), and most of the others score low."""
    from velox_b200.csrc import ops
    rng = np.random.default_rng(D + window)
    T, S, eps, scale = 2 * window + 45, 16, 1e-5, 6.0 / D
    base = rng.normal(size=(T, G, D)) * rng.uniform(0.2, 4.0, size=(T, G, 1))
    k, v = bf(base), bf(rng.normal(size=(T, G, Dv)))
    q = rng.normal(size=(T, H, D))
    for t in range(T):
        j = t - (window - 1) if t % 2 else t - window     # odd rows ask for the last key they see, even rows for the first they do not
        if j >= 0:
            q[t] = np.repeat(k[j], H // G, axis=0) * 1.5
    q = bf(q)
    store = (lambda x: x) if dtype == torch.float32 else bf
    qn, kn = store(P.unit_rms(q, eps)), store(P.unit_rms(k, eps))
    mask = P.window_mask(T, window)
    want = np.stack([P.softmax((qn[:, n] @ kn[:, n // (H // G)].T) * scale, mask, plus_one=True) @ v[:, n // (H // G)] for n in range(H)], axis=1)
    wrong = np.stack([P.softmax((qn[:, n] @ kn[:, n // (H // G)].T) * scale, P.window_mask(T, window + 1), plus_one=True) @ v[:, n // (H // G)] for n in range(H)], axis=1)
    assert np.abs(want - wrong).max() > 0.3               # (one token off shows)
    want = want.reshape(T, -1)
    x = dev(np.concatenate([a.reshape(T, -1) for a in (q, k, v)], 1), dtype)
    pages = -(-T // S)
    order = rng.permutation(pages + 3)[:pages]
    kp = torch.full((pages + 3, G, S, D), float("nan"), dtype=dtype, device=DEV)
    vp = torch.full((pages + 3, G, S, Dv), float("nan"), dtype=dtype, device=DEV)
    one = torch.ones(D, device=DEV)
    ops.qk_norm_rope_kv(x, one, one, eps, None, 0, ints(range(T)), ints(order[t // S] * S + t % S for t in range(T)), kp, vp, H, G, D, Dv)
    close(x[:, :H * D], qn.reshape(T, -1), TOL[dtype])
    more = dict(sinks=torch.zeros(H, device=DEV))
    table = ints(order).view(1, -1).contiguous()
    got = ops.paged_attention_generic(x, x.shape[1], kp, vp, table, ints([0] * T), ints(range(T)), scale, window, H, G, D, T, v_head_dim=Dv, **more)
    close(got, want, TOL[dtype])
    if not ops.biased_attention_supported(dtype, D, Dv, S):
        return
    for lo in (0, 1, T - 20, window):
        part = x[lo:].contiguous()
        got = ops.biased_prefill_attention(part, x.shape[1], kp, vp, table, ints([0, T - lo]), ints([lo]), scale, window, 0, 0.0, H, G, D, Dv, 1,
                                           T - lo, T - lo, **more)
        close(got, want[lo:], TOL[dtype])
    got = ops.biased_decode_attention(x, x.shape[1], kp, vp, table, ints([0] * T), ints(range(T)), scale, window, 0, 0.0, H, G, D, Dv, T, max_kv=T, **more)
    close(got, want, TOL[dtype])
    if D == Dv and ops.prefill_attention_tc_supported(dtype, D, S, H // G):
        got = ops.paged_prefill_attention_tc(x, x.shape[1], kp, vp, table, ints([0, T]), ints([0]), scale, window, H, G, D, 1, T, T, halves=True, **more)
        close(got, want, TOL[dtype])


# -- experts -------------------------------------------------------------------------------------------------------------------

def decided(h, W, router, least=1e-3):
    return h[P.router_margins(h, W, router) > least]


@pytest.mark.parametrize("n,top,groups", [(8, 3, (4, 2)), (6, 2, (2, 1)), (12, 4, (3, 2)), (5, 2, (5, 3)), (6, 6, None), (64, 6, (8, 4)), (200, 8, (10, 3)), (1, 1, None)])
@pytest.mark.parametrize("T,E", [(70, 64), (40, 30), (33, 2048)])
def test_routing_by_pairs_of_group_scores(n, top, groups, T, E):
    from velox_b200.csrc import ops
    rng = np.random.default_rng(n)
    router = {"experts": n, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    W = rng.normal(size=(n, E)) * 2.0 / np.sqrt(E)
    h = decided(rng.normal(size=(3 * T, E)), W, router)[:T]
    assert len(h) > 10
    chosen, weight = P.route(h, W, router)
    g, keep = groups or (1, 1)
    plan = ops.moe_route(dev(h), dev(W), None, n, top, scores="sigmoid", groups=g, keep_groups=keep, group_pair=True, renormalise=True)
    assert np.array_equal(np.sort(plan.chosen.view(len(h), top).cpu().numpy(), 1), np.sort(chosen, 1))
    order = np.argsort(plan.chosen.view(len(h), top).cpu().numpy(), 1)
    close(torch.from_numpy(np.take_along_axis(plan.weight.cpu().numpy(), order, 1)), np.take_along_axis(weight, np.argsort(chosen, 1), 1), 1e-5)


def test_a_group_of_two_good_experts_beats_one_with_the_best():
    from velox_b200.csrc import ops
    z = np.array([[3.0, -3.0, 1.0, 0.9, 0.0, 0.0], [0.0, 0.1, 40.0, -40.0, 2.0, 2.5]])
    plan = ops.moe_route(dev(z), dev(np.eye(6)), None, 6, 2, scores="sigmoid", groups=3, keep_groups=1, group_pair=True, renormalise=True)
    assert plan.chosen.view(2, 2).cpu().tolist() == [[2, 3], [5, 4]]
    plain = ops.moe_route(dev(z), dev(np.eye(6)), None, 6, 2, scores="sigmoid", groups=3, keep_groups=1)
    assert plain.chosen.view(2, 2).cpu().tolist() == [[0, 1], [2, 3]]
    close(plan.weight.sum(1), np.ones(2), 1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E,I,n,top,groups,limit", [(1, 64, 32, 6, 2, (3, 2), 1.0), (7, 72, 20, 4, 4, None, 0.5), (70, 128, 64, 6, 3, (2, 1), 2.0),
                                                      (300, 64, 24, 12, 3, (4, 2), 1.5), (1100, 128, 64, 8, 2, (4, 2), 0.8), (600, 256, 512, 4, 2, (2, 2), 3.0),
                                                      (9, 40, 10, 3, 3, None, 1.2), (2000, 128, 136, 5, 4, None, 1.0)])
def test_experts_with_a_bounded_gate(dtype, T, E, I, n, top, groups, limit):
    """Every grouped product (multiply-adds, row tiles of 64 and of 16 on the tensor cores, tcgen05 with both tile widths, inner sizes
    that are no multiple of 8) through the part; gates and ups of several times the limit on either side."""
    from velox_b200.parts import PartSpec, Runtime, build_part
    rng = np.random.default_rng(T)
    router = {"experts": n, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    W = {"router": bf(rng.normal(size=(n, E)) * 2.0 / np.sqrt(E))}
    for e in range(n):
        for x in ("gate", "up"):
            W["e%d.%s" % (e, x)] = bf(rng.normal(size=(I, E)) * 2.0 / np.sqrt(E))
        W["e%d.down" % e] = bf(rng.normal(size=(E, I)) / np.sqrt(I))
    h = decided(bf(rng.normal(size=(4 * T + 20, E))), W["router"], router)[:T]
    part = build_part("feed_forward", PartSpec("routed_experts", "", dict(
        hidden_size=E, experts=n, top=top, intermediate_size=I, router_bias=False, scores="sigmoid", groups=(groups or (1, 1))[0],
        keep_groups=(groups or (1, 1))[1], group_pair=True, renormalise=True, capped=(limit, 1.702))))
    assert {s.name: s.shape for s in part.tensor_specs()} == {k: v.shape for k, v in W.items()}
    part.bind({k: dev(v, torch.float32 if k == "router" else dtype) for k, v in W.items()}, Runtime(dtype, torch.device(DEV)))
    m = {"router": router, "expert": {"ff": I, "limit": limit}}
    exact = P.routed_feed_forward(h, W, m)
    got = part.forward(dev(h, dtype))
    if dtype == torch.float32:
        close(got, exact, 2e-5)
    else:
        cost = np.abs(P.routed_feed_forward(h, W, m, store=bf) - exact).max()
        assert np.abs(host(got) - exact).max() <= 2.0 * cost

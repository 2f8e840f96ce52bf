"""The kernels behind Negilorn's mechanisms, each alone against its plain function (`plain_negilorn.py`): token shift fused
with the residual update and the norm (with and without the mixes of a second shift), the second shift alone, decays through a
narrow middle, the recurrence with a bonus (single tokens, portions, stretches side by side), the norm per head with a weight
per channel, projections with an input each, attention over chunks with one added to the denominator in every kernel with a
key that stands out just inside and just outside a chunk's edge, rotation stretched by wavelength and of queries alone,
routing by sigmoids, experts without a gate whose weight enters before the activation, and the plain activation on the
matrix products' sums."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_negilorn as N

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
TOL = {torch.float32: 2e-5, torch.bfloat16: 8e-3}   # (a bfloat16 result is rounded once: 2^-8 of its size)


def dev(x, dtype=torch.float32):
    return torch.from_numpy(np.array(x, dtype=np.float64, order="C")).to(DEV).to(dtype)


def ints(x):
    return torch.tensor(list(x), dtype=torch.int32, device=DEV)


def bf(x):
    return N.store_bfloat16(x)


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def close(got, want, tol):
    got = host(got)
    scale = max(1.0, float(np.abs(want).max()))
    assert got.shape == want.shape and np.isfinite(got).all()
    assert np.abs(got - want).max() <= tol * scale, "largest error %g of scale %g" % (np.abs(got - want).max(), scale)


def step_of(lens, slots):
    """The fields of a step's context that the shift kernels read."""
    cu = np.concatenate([[0], np.cumsum(lens)])
    return SimpleNamespace(n_seqs=len(lens), max_new=max(lens), cu_seqlens=ints(cu), state_slots=ints(slots), new_lens=list(lens),
                           seq_of_token=ints(np.repeat(np.arange(len(lens)), lens)), positions=ints(np.zeros(sum(lens))))


def rows_of(lens):
    cu = np.concatenate([[0], np.cumsum(lens)])
    return [slice(int(a), int(b)) for a, b in zip(cu[:-1], cu[1:])]


# -- token shift -----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,k", [(72, 0), (72, 5), (30, 3), (128, 5), (1000, 0), (2048, 5), (2052, 1), (4100, 2), (8200, 0), (1030, 4)])
@pytest.mark.parametrize("with_delta", [True, False])
def test_residual_update_norm_shift_and_mixes_in_one_pass(dtype, E, k, with_delta):
    """Three sequences through steps of unequal portions (single rows, rows of many, one left out of a step) against the whole
    sequences at once; slots hold the last rows between the steps and nothing else is carried."""
    from velox_b200.csrc import ops
    rng = np.random.default_rng(E + k)
    lens = [23, 9, 40]
    x = [rng.normal(size=(n, E)) for n in lens]
    d = [bf(rng.normal(size=(n, E))) if with_delta else np.zeros((n, E)) for n in lens]
    mu, nu, g = rng.uniform(size=E), rng.uniform(size=(max(k, 1), E)), 1.3
    x = [host(dev(a)) for a in x]
    total = [a + b for a, b in zip(x, d)]
    n = [N.scalar_norm(t, g, 1e-5) for t in total]
    h = [N.token_shift(a, mu) for a in n]
    want = h if not k else [np.stack([N.token_shift(a, nu[i]) for i in range(k)]) for a in h]
    slots = [2, 0, 3]
    st_n, st_h = torch.zeros((4, E), device=DEV), torch.zeros((4, E), device=DEV)
    st_n[1], st_h[1] = 5.0, 5.0
    at = [0, 0, 0]
    for plan in ([5, 1, 2], [1, 1, 1], [0, 2, 33], [16, 5, 0], [1, 0, 4]):
        who = [i for i in range(3) if plan[i]]
        ls = [plan[i] for i in who]
        ctx = step_of(ls, [slots[i] for i in who])
        piece = lambda a: np.concatenate([a[i][at[i]:at[i] + plan[i]] for i in who])
        res, delta = dev(piece(x)), dev(piece(d), dtype) if with_delta else None
        before = res.clone()
        out_x, out = ops.shift_norm(res, delta, torch.full((E,), g, device=DEV), 1e-5, dev(mu), ctx, st_n, dtype,
                                    mixes=dev(nu) if k else None, mix_state=st_h if k else None)
        assert torch.equal(res, before) and (out_x is res) == (not with_delta)
        close(out_x, piece(total), 1e-6)
        w = np.concatenate([want[i][..., at[i]:at[i] + plan[i], :] for i in who], axis=-2)
        close(out, w, TOL[dtype])
        for i in who:
            at[i] += plan[i]
            close(st_n[slots[i]], n[i][at[i] - 1], 1e-5)
            if k:
                close(st_h[slots[i]], h[i][at[i] - 1], 1e-5)
    assert at == lens and float(st_n[1].min()) == 5.0 == float(st_h[1].max())
    if not k:
        assert float(st_h[2].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("k", [0, 5])
def test_requests_that_lie_in_many_blocks_of_rows_are_cut_anywhere_with_the_same_bits(dtype, k):
    """5,000 rows in one step (several rows a block; requests of 1, 2 and 3 rows between long ones, so that blocks hold the end
    of one request, a whole one and the start of the next) against the same requests alone and in portions: every bit."""
    from velox_b200.csrc import ops
    rng = np.random.default_rng(k)
    E, lens = 64, [1700, 1, 2, 3, 900, 1, 1, 2000, 2, 390]
    res, delta = dev(rng.normal(size=(sum(lens), E))), dev(rng.normal(size=(sum(lens), E)), dtype)
    w, mu, nu = dev(1.0 + 0.1 * rng.normal(size=E)), dev(rng.uniform(size=E)), dev(rng.uniform(size=(5, E)))

    def run(r, d, ctx, sn, sh):
        return ops.shift_norm(r, d, w, 1e-5, mu, ctx, sn, dtype, mixes=nu if k else None, mix_state=sh if k else None)
    sn, sh = torch.zeros((12, E), device=DEV), torch.zeros((12, E), device=DEV)
    slots = [11 - i for i in range(len(lens))]
    x_all, h_all = run(res, delta, step_of(lens, slots), sn, sh)
    for i, rows in enumerate(rows_of(lens)):
        for cuts in ([lens[i]], [c for c in (1, 700, 3) if sum((1, 700, 3)) < lens[i]] + [lens[i] - (704 if lens[i] > 704 else 0)]):
            sn1, sh1 = torch.zeros((12, E), device=DEV), torch.zeros((12, E), device=DEV)
            at, got = rows.start, []
            for c in cuts:
                x1, h1 = run(res[at:at + c].contiguous(), delta[at:at + c].contiguous(), step_of([c], [slots[i]]), sn1, sh1)
                assert torch.equal(x1, x_all[at:at + c])
                got.append(h1)
                at += c
            assert torch.equal(torch.cat(got, dim=-2), h_all[..., rows, :])
            assert torch.equal(sn1[slots[i]], sn[slots[i]]) and torch.equal(sh1[slots[i]], sh[slots[i]])
    total = host(res) + host(delta)
    for i in (0, 4, 9):
        rows = rows_of(lens)[i]
        n = N.unit_rms(total[rows], 1e-5) * host(w)
        h = N.token_shift(n, host(mu))
        want = np.stack([N.token_shift(h, v) for v in host(nu)]) if k else h
        close(h_all[..., rows, :], want, TOL[dtype])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E", [40, 1536])
def test_the_second_shift_alone(dtype, E):
    from velox_b200.csrc import ops
    rng = np.random.default_rng(E)
    lens, nu = [13, 30], rng.uniform(size=(3, E))
    h = [bf(rng.normal(size=(n, E))) for n in lens]
    want = [np.stack([N.token_shift(a, nu[i]) for i in range(3)]) for a in h]
    state, at = torch.zeros((2, E), device=DEV), [0, 0]
    for plan in ([4, 1], [1, 1], [8, 28]):
        out = ops.shift_mix(dev(np.concatenate([h[i][at[i]:at[i] + plan[i]] for i in (0, 1)]), dtype), dev(nu), step_of(plan, [1, 0]), state)
        close(out, np.concatenate([want[i][:, at[i]:at[i] + plan[i]] for i in (0, 1)], axis=1), TOL[dtype])
        at = [a + p for a, p in zip(at, plan)]
        close(state[1], h[0][at[0] - 1], 0.0)
        close(state[0], h[1][at[1] - 1], 0.0)


# -- time mixing -----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("rank,C", [(1, 37), (5, 256), (16, 300), (64, 2048), (130, 72)])
def test_decays_through_a_narrow_middle(rank, C):
    from velox_b200.csrc import ops
    rng = np.random.default_rng(rank)
    w2, w0 = bf(rng.normal(size=(C, rank)) / np.sqrt(rank)), bf(rng.normal(-2.0, 1.5, C))
    for T in (1, 2, 7, 16, 17, 45):
        low = rng.normal(size=(T, rank)) * 2.0
        wide = dev(np.concatenate([rng.normal(size=(T, 3)), low], 1))
        got = ops.low_rank_decay(wide[:, 3:], dev(w2.T), dev(w0))
        want = np.log(N.wkv_decay(host(wide)[:, 3:], {"w1": np.eye(rank), "w2": w2, "w0": w0}))
        assert np.abs(host(got) / want - 1.0).max() < 1e-5


def mixing_case(rng, T, H, D):
    r, k, v = (bf(rng.normal(size=(T, H, D))) for _ in range(3))
    log_w = -np.exp(rng.normal(-2.5, 1.5, (T, H, D)))
    log_w[:, :, 0] = -1e-4                   # a channel that forgets next to nothing: the first key stays in it for good
    log_w[:, :, D - 1] = -40.0               # and one that keeps nothing but the token before
    return r, k, v, host(dev(log_w)), bf(rng.normal(size=(H, D)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D", [(3, 12), (2, 20), (4, 32), (2, 64), (1, 100), (2, 128), (1, 200), (1, 8)])
def test_the_recurrence_with_a_bonus_token_by_token_in_portions_and_in_stretches(dtype, H, D):
    """A request of 700 tokens, whole in stretches side by side, in portions and as single tokens beside another request, always
    against the plain walk; the columns of r, k, v lie in one row or in matrices of their own.  The first token's key is made
    large: the channel that forgets nothing carries it to the end."""
    from velox_b200.csrc import ops
    rng = np.random.default_rng(D)
    T, HD = 700, H * D
    r, k, v, log_w, u = mixing_case(rng, T, H, D)
    k[0, :, 0] = 20.0
    want, S = N.wkv_walk(r, k, v, np.exp(log_w), u)
    with_first, _ = N.wkv_walk(r, np.concatenate([0 * k[:1], k[1:]]), v, np.exp(log_w), u)
    assert np.abs(want[-1] - with_first[-1]).max() > 0.5
    tol = 4e-5
    bonus, lw = dev(u), dev(log_w.reshape(T, HD))

    def rows(a, b, packed):
        parts = [z[a:b].reshape(b - a, HD) for z in (r, k, v)]
        if packed:
            return dev(np.concatenate(parts + [np.zeros((b - a, 3))], 1), dtype), (0, HD, 2 * HD)
        return dev(np.stack(parts), dtype), (0, (b - a) * HD, 2 * (b - a) * HD)

    def walk(a, b, state, packed, stretches=None):
        x, cols = rows(a, b, packed)
        return ops.linear_attention_walk(x, *cols, state, ints([0, b - a]), ints([1]), 1, H, D, D, gate=lw[a:b], gate_is_log=True, bonus=bonus,
                                         stretches=stretches)
    for packed in (False, True):
        state = torch.zeros((3, H, D, D), device=DEV)
        close(walk(0, T, state, packed), want.reshape(T, HD), tol)
        close(state[1], S, tol)
        state.zero_()
        got = [walk(0, 300, state, packed, ops.StretchPlan([300], DEV)), walk(300, 301, state, packed), walk(301, 303, state, packed),
               walk(303, T, state, packed, ops.StretchPlan([T - 303], DEV, 64))]
        close(torch.cat(got), want.reshape(T, HD), tol)
        close(state[1], S, tol)
        assert float(state[0].abs().max()) == 0.0 == float(state[2].abs().max())
    # decoding beside another request: two single tokens a step
    state = torch.zeros((3, H, D, D), device=DEV)
    for t in range(12):
        x = dev(np.stack([np.concatenate([z[j].ravel() for z in (r, k, v)]) for j in (t, t + 100)]), dtype)
        got = ops.linear_attention_walk(x, 0, HD, 2 * HD, state, ints([0, 1, 2]), ints([2, 0]), 2, H, D, D,
                                        gate=torch.stack([lw[t], lw[t + 100]]), gate_is_log=True, bonus=bonus)
        close(got[0], want[t].reshape(HD), tol)
        if t == 0:
            close(got[1], (r[100] * u * k[100]).sum(-1, keepdims=True).repeat(D, -1).reshape(HD) * v[100].reshape(HD), tol)


@pytest.mark.parametrize("H,D", [(3, 12), (2, 32), (4, 64), (2, 128), (1, 100)])
def test_the_norm_per_head_takes_a_weight_per_channel(H, D):
    from velox_b200.csrc import ops
    rng = np.random.default_rng(D)
    for T in (1, 5, 70):
        o, g, w, shared = rng.normal(size=(T, H * D)), bf(rng.normal(size=(T, H * D + 8))), 1.0 + rng.normal(size=H * D), 1.0 + rng.normal(size=D)
        for gate_dtype, out_dtype in ((torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16), (torch.float32, torch.bfloat16)):
            for act, name in ((N.silu, "silu"), (N.sigmoid, "sigmoid")):
                for weight, full in ((w, w), (shared, np.tile(shared, H)), (None, np.ones(H * D))):
                    got = ops.head_norm_gate(dev(o), dev(g, gate_dtype)[:, 8:], None if weight is None else dev(weight), H, 1e-5, name, out_dtype=out_dtype)
                    assert got.dtype == out_dtype
                    want = N.unit_rms(o.reshape(T, H, D), 1e-5).reshape(T, H * D) * full * act(g[:, 8:])
                    close(got, want, TOL[out_dtype])


@pytest.mark.parametrize("M", [1, 3, 8])
@pytest.mark.parametrize("seg,last,K", [(60, 5, 64), (256, 16, 256), (32, 64, 96), (2048, 64, 2048), (8, 1, 32), (16, 16, 160)])
def test_projections_with_an_input_each_in_one_launch(M, seg, last, K):
    from velox_b200.csrc import ops
    rng = np.random.default_rng(seg)
    xs, w = bf(rng.normal(size=(5, M, K))), bf(rng.normal(size=(4 * seg + last, K)) / np.sqrt(K))
    want = np.concatenate([xs[i] @ w[i * seg:(i + 1) * seg if i < 4 else None].T for i in range(5)], axis=1)
    for out_dtype in (torch.float32, torch.bfloat16):
        close(ops.gemm_inputs(dev(xs, torch.bfloat16), dev(w, torch.bfloat16), seg, out_dtype), want, TOL[out_dtype])
    for dtype in (torch.float32, torch.bfloat16):
        got = ops.gemm_members(dev(xs[:4], dtype), dev(w[:4 * seg].reshape(4, seg, K), dtype))
        close(got, np.stack([xs[i] @ w[i * seg:(i + 1) * seg].T for i in range(4)]), TOL[dtype])


# -- attention over chunks ---------------------------------------------------------------------------------------------------

def paged(k, v, page_size, n_pages, seed):
    """Keys [T, G, D] and values [T, G, Dv] into NaN-filled pools through a scattered table."""
    T = k.shape[0]
    table = np.random.default_rng(seed).permutation(n_pages)[:-(-T // page_size)]
    kp = np.full((n_pages, k.shape[1], page_size, k.shape[2]), np.nan)
    vp = np.full((n_pages, v.shape[1], page_size, v.shape[2]), np.nan)
    for j in range(T):
        kp[table[j // page_size], :, j % page_size] = k[j]
        vp[table[j // page_size], :, j % page_size] = v[j]
    return kp, vp, table


def chunked_attention(q, k, v, scale, chunk, cap, gates):
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        p = N.softmax_plus_one(N.bounded((q[:, h] @ k[:, g].T) * scale, cap), N.chunk_mask(T, chunk))
        out[:, h] = p @ v[:, g] * N.sigmoid(gates[:, h:h + 1])
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv,chunk,cap", [(4, 2, 10, 12, 7, 5.0), (4, 2, 64, 64, 100, 20.0), (2, 1, 128, 64, 50, 0.0), (6, 2, 32, 32, 96, 12.0),
                                                (3, 3, 80, 80, 16, 8.0), (5, 1, 96, 96, 33, 8.0), (2, 2, 64, 128, 1, 6.0), (8, 2, 128, 128, 300, 15.0),
                                                (4, 1, 24, 24, 0, 9.0), (2, 1, 64, 32, 0, 0.0)])
def test_attention_over_chunks_in_every_kernel(dtype, H, G, D, Dv, chunk, cap):
    """600 positions in one portion, in a late portion whose earlier pages are gone, as single tokens with their keys in one run
    and in several.  For the last query of every chunk the chunk's first key is made to stand out (it is seen from the far end of
    the chunk), and for the first query of every chunk the key right before it (which the edge hides: such a query sees itself
    alone, with a weight below one)."""
    from velox_b200.csrc import ops
    rng = np.random.default_rng(H * D + chunk)
    T, S = 600, 16
    scale = 1.0 / np.sqrt(D)
    q, k, v, gates = bf(rng.normal(size=(T, H, D))), bf(rng.normal(size=(T, G, D))), bf(rng.normal(size=(T, G, Dv))), bf(rng.normal(size=(T, H)))
    step = chunk or T
    for c in range(0, T, step):
        last = min(c + step, T) - 1
        for h in range(H):
            kk = k[c, h // (H // G)]
            if last > c:
                q[last, h] = bf(8.0 * kk / np.sqrt(np.mean(kk ** 2)))
            if c and step > 1:
                kk = k[c - 1, h // (H // G)]
                q[c, h] = bf(8.0 * kk / np.sqrt(np.mean(kk ** 2)))
    want = chunked_attention(q, k, v, scale, chunk, cap, gates)
    if chunk > 1 and cap == 0.0:
        assert np.abs(want[chunk - 1, 0] / N.sigmoid(gates[chunk - 1, 0]) - v[0, 0]).max() < 0.05
    want = want.reshape(T, -1)
    kp, vp, table = paged(k, v, S, 45, 1)
    k_pool, v_pool = dev(kp, dtype), dev(vp, dtype)
    pad = (-(H * D + H)) % 8
    x = dev(np.concatenate([q.reshape(T, -1), gates, np.zeros((T, pad))], 1), dtype)
    zeros = torch.zeros(H, device=DEV)
    more = dict(sinks=zeros, gate_col=H * D, softcap=cap, chunk=chunk)

    def table_from(first_query):
        bt = torch.full((1, 45), -1, dtype=torch.int32, device=DEV)
        first = (first_query - first_query % chunk) // S if chunk else 0
        bt[0, first:len(table)] = ints(table[first:])
        return bt
    # a table entry of -1 names no page: a kernel that read one would leave the pool (the general kernel and the prompt kernel clamp
    # hidden keys onto visible ones)
    for lo in (0, 537, T - 40):
        xs, n = x[lo:].contiguous(), T - lo
        got = ops.paged_attention_generic(xs, xs.shape[1], k_pool, v_pool, table_from(lo), ints([0] * n), ints(range(lo, T)), scale, 0, H, G, D, n,
                                          v_head_dim=Dv, **more)
        close(got, want[lo:], TOL[dtype])
        if ops.biased_attention_supported(dtype, D, Dv, S):
            got = ops.biased_prefill_attention(xs, xs.shape[1], k_pool, v_pool, table_from(lo), ints([0, n]), ints([lo]), scale, 0, 0, 0.0, H, G, D,
                                               Dv, 1, n, n, **more)
            close(got, want[lo:], TOL[dtype])
    if not ops.biased_attention_supported(dtype, D, Dv, S):
        return
    edges = sorted({t for c in range(step, T, step) for t in (c - 1, c, c + 1) if t < T} | {0, 1, 15, 16, T - 1})[:40]
    for max_kv in (0, T):   # (the bound on the keys is what asks for runs)
        rows = torch.stack([x[t] for t in edges]).contiguous()
        got = ops.biased_decode_attention(rows, rows.shape[1], k_pool, v_pool, table_from(0), ints([0] * len(edges)), ints(edges), scale, 0, 0, 0.0,
                                          H, G, D, Dv, len(edges), max_kv=max_kv, **more)
        close(got, want[edges], TOL[dtype])
        one = ops.biased_decode_attention(x[T - 1:].contiguous(), x.shape[1], k_pool, v_pool, table_from(T - 1), ints([0]), ints([T - 1]), scale, 0, 0,
                                          0.0, H, G, D, Dv, 1, max_kv=max_kv, **more)
        close(one, want[T - 1:], TOL[dtype])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv,rot", [(4, 2, 10, 12, 6), (2, 1, 64, 64, 32), (4, 2, 128, 128, 128), (5, 1, 72, 33, 26), (1, 1, 200, 64, 200)])
@pytest.mark.parametrize("T", [5, 130])
def test_rotation_stretched_by_wavelength_with_and_without_keys(dtype, H, G, D, Dv, rot, T):
    """Queries and keys turned and written; and a row of queries alone (a layer that borrows its keys), behind which the gates' columns
    stay as they are."""
    from velox_b200.csrc import ops
    from velox_b200.parts.position import RotaryPosition
    rng = np.random.default_rng(D)
    sc = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}
    q, k, v = bf(rng.normal(size=(T, H, D))), bf(rng.normal(size=(T, G, D))), bf(rng.normal(size=(T, G, Dv)))
    pos = np.arange(T) + 700
    spec = {"base": 300.0, "dims": rot, "scaling": sc}
    part = RotaryPosition("", head_dim=D, theta=300.0, rotary_dim=rot, scaling=sc)
    inv = part.rotary_table(DEV)[0]
    want_q, want_k = N.rotate_half(q, pos, spec), N.rotate_half(k, pos, spec)
    tol = max(TOL[dtype], 1e-4)   # (a float32 angle of some 800 radians is good to 5e-5)
    S, extra = 16, 8 + (-(H * D)) % 8
    x = dev(np.concatenate([q.reshape(T, -1), np.full((T, extra), 7.0)], 1), dtype)
    ops.qk_norm_rope_kv(x, None, None, 1e-5, inv, rot, ints(pos), None, None, None, H, 0, D, Dv)
    close(x[:, :H * D], want_q.reshape(T, -1), tol)
    assert (x[:, H * D:] == 7.0).all()
    x = dev(np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), np.full((T, extra), 7.0)], 1), dtype)
    kp = torch.full((10, G, S, D), float("nan"), dtype=dtype, device=DEV)
    vp = torch.full((10, G, S, Dv), float("nan"), dtype=dtype, device=DEV)
    ops.qk_norm_rope_kv(x, None, None, 1e-5, inv, rot, ints(pos), ints(range(T)), kp, vp, H, G, D, Dv)
    close(x[:, :H * D], want_q.reshape(T, -1), tol)
    for j in (0, T - 1):
        close(kp[j // S, :, j % S], want_k[j], tol)
        close(vp[j // S, :, j % S], v[j], 0.0)


# -- experts -----------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E,I,n,top,shared", [(1, 64, 32, 5, 2, True), (7, 72, 20, 4, 4, False), (70, 128, 64, 6, 1, True), (300, 64, 24, 12, 3, True),
                                                (1100, 128, 64, 7, 2, True), (600, 256, 512, 4, 2, False), (9, 40, 10, 3, 3, True), (5, 64, 16, 1, 1, True)])
def test_experts_without_a_gate_weighted_on_their_input(dtype, T, E, I, n, top, shared):
    """Every grouped product (multiply-adds, row tiles of 64 and of 16 on the tensor cores, tcgen05 with both tile widths) through the
    part, beside the plain sum; one expert's scores are tiny, so that its weight on the wrong side of the square would show."""
    from velox_b200.parts import PartSpec, Runtime, build_part
    rng = np.random.default_rng(T)
    P = {"router": bf(rng.normal(size=(n, E)) * 2.0 / np.sqrt(E))}
    for e in range(n):
        P["e%d.up" % e], P["e%d.down" % e] = bf(rng.normal(size=(I, E)) / np.sqrt(E)), bf(rng.normal(size=(E, I)) / np.sqrt(I))
    if shared:
        P["shared.up"], P["shared.down"] = bf(rng.normal(size=(2 * I, E)) / np.sqrt(E)), bf(rng.normal(size=(E, 2 * I)) / np.sqrt(2 * I))
    h = bf(rng.normal(size=(4 * T, E)))
    h = h[N.router_margins(h, P["router"], top) > 1e-3][:T]
    part = build_part("feed_forward", PartSpec("routed_experts", "", dict(
        hidden_size=E, experts=n, top=top, intermediate_size=I, activation="relu2", router_bias=False, names=("up", "down"), scores="sigmoid",
        gated=False, weight_input=True, shared=PartSpec("dense_mlp", "shared.", dict(
            hidden_size=E, intermediate_size=2 * I, activation="relu2", names=("up", "down"))) if shared else None)))
    assert {s.name: s.shape for s in part.tensor_specs()} == {k: v.shape for k, v in P.items()}
    part.bind({k: dev(v, torch.float32 if k == "router" else dtype) for k, v in P.items()}, Runtime(dtype, torch.device(DEV)))
    m = {"router": {"experts": n, "top": top}, "shared": {"ff": 2 * I} if shared else None}
    want = N.routed_feed_forward(h, P, m)
    got = part.forward(dev(h, dtype))
    if dtype == torch.float32:
        close(got, want, 2e-5)
    else:
        cost = np.sqrt(np.mean(np.square(N.routed_feed_forward(h, P, m, store=N.store_bfloat16) - want)))
        assert np.isfinite(host(got)).all() and np.sqrt(np.mean(np.square(host(got) - want))) < 1.3 * cost


def test_routing_by_sigmoids_takes_the_largest_logits_even_where_the_sigmoid_is_one():
    from velox_b200.csrc import ops
    rng = np.random.default_rng(3)
    T, E, n, top = 50, 64, 9, 3
    W = rng.normal(size=(n, E))
    h = bf(rng.normal(size=(T, E)) * 6.0)         # (logits of some tens: the float32 sigmoid is exactly 1 from 17 on)
    h = h[N.router_margins(h, W, top) > 1e-2]
    plan = ops.moe_route(dev(h), dev(W), None, n, top, scores="sigmoid")
    order = np.argsort(-(h @ W.T), axis=1)[:, :top]
    assert np.array_equal(plan.chosen.view(-1, top).cpu().numpy(), order)
    s = N.sigmoid(h @ W.T)
    assert np.abs(host(plan.weight) - np.take_along_axis(s, order, 1)).max() < 2e-6
    # with a correction the choice is by the corrected score and the weight stays the score
    corr = rng.normal(size=n)
    plan = ops.moe_route(dev(h), dev(W), None, n, top, scores="sigmoid", correction=dev(corr), route_scale=1.5)
    order = np.argsort(-(s + host(dev(corr))), axis=1, kind="stable")[:, :top]
    assert np.array_equal(np.sort(plan.chosen.view(-1, top).cpu().numpy(), 1), np.sort(order, 1))
    assert np.abs(np.sort(host(plan.weight), 1) - np.sort(1.5 * np.take_along_axis(s, order, 1), 1)).max() < 3e-6


@pytest.mark.parametrize("M,n,K", [(3, 40, 64), (8, 256, 128), (130, 256, 192), (2048, 2560, 256), (200, 128, 64)])
def test_the_plain_activation_on_the_sums_of_the_matrix_products(M, n, K):
    from velox_b200.csrc import ops
    rng = np.random.default_rng(M)
    a, w = bf(rng.normal(size=(M, K))), bf(rng.normal(size=(n, K)) / np.sqrt(K))
    z = a @ w.T
    A, W = dev(a, torch.bfloat16), dev(w, torch.bfloat16)
    for name, fn in (("relu2", N.squared_relu), ("relu", lambda t: np.maximum(t, 0.0)), ("silu", N.silu)):
        if ops.skinny_supported(M, K, A, W):
            close(ops.gemm_skinny(A, W, None, torch.bfloat16, activation=name), fn(z), TOL[torch.bfloat16])
        close(ops.act(dev(z), name, out_dtype=torch.bfloat16), fn(z), TOL[torch.bfloat16])
        if ops.tcgen05_supported(A, W) and name in ops.TCGEN05_ACTIVATIONS:
            for wide in (True, False):
                close(ops.gemm_tcgen05(A, W, None, activation=name, wide=wide), fn(z), TOL[torch.bfloat16])
    ops.check_device_errors()
    with pytest.raises(ops.KernelError):
        ops.gemm_tcgen05(A, W, None, activation="silu")


def test_a_norm_with_one_number_multiplies_every_channel():
    from velox_b200.parts import PartSpec, Runtime, build_part
    rng = np.random.default_rng(0)
    norm = build_part("norm", PartSpec("rms_norm", "n", dict(size=72, eps=1e-5, weight_name="", scalar=True)))
    assert [(s.name, s.shape) for s in norm.tensor_specs()] == [("n", ())]
    norm.bind({"n": torch.tensor(0.7, device=DEV)}, Runtime(torch.float32, torch.device(DEV)))
    x = rng.normal(size=(5, 72))
    close(norm.add_norm(dev(x), None), N.scalar_norm(x, 0.7, 1e-5), 1e-5)


def test_the_time_mixing_makes_its_own_mixes_under_another_block():
    """`wkv` called like any mixer (`forward`) gives what the block's fused kernel and `forward_mixed` give."""
    from velox_b200.cache.manager import CacheManager
    from velox_b200.parts import PartSpec, Runtime, build_part
    rng = np.random.default_rng(1)
    E, H, D, rank, lens = 48, 3, 16, 6, [11, 20]
    P = {"mu." + x: bf(rng.uniform(size=E)) for x in "rkvgw"}
    P.update({x: bf(rng.normal(size=(H * D, E)) / np.sqrt(E)) for x in "rkvg"})
    P.update({"o": bf(rng.normal(size=(E, H * D)) / np.sqrt(H * D)), "w1": bf(rng.normal(size=(rank, E)) / np.sqrt(E)),
              "w2": bf(rng.normal(size=(H * D, rank))), "w0": bf(rng.normal(-2, 1, H * D)), "u": bf(rng.normal(size=(H, D))),
              "norm": bf(1 + 0.2 * rng.normal(size=H * D))})
    part = build_part("mixer", PartSpec("wkv", "m.", dict(hidden_size=E, num_heads=H, head_dim=D, eps=1e-5)))
    assert {s.name for s in part.tensor_specs()} == {"m." + k for k in P}
    part.bind({"m." + k: dev(v) for k, v in P.items()}, Runtime(torch.float32, torch.device(DEV)))
    cache = CacheManager([part.cache_spec()], [None], 16, 2, 2, 2, device=torch.device(DEV))
    h = [rng.normal(size=(n, E)) for n in lens]
    want = [N.wkv(a, P, {"heads": H, "dim": D}, 1e-5) for a in h]
    at = [0, 0]
    for plan in ([3, 1], [1, 1], [7, 18]):
        got = part.forward(dev(np.concatenate([h[i][at[i]:at[i] + plan[i]] for i in (0, 1)])), step_of(plan, [1, 0]), cache.layer(0))
        close(got, np.concatenate([want[i][at[i]:at[i] + plan[i]] for i in (0, 1)]), 5e-5)
        at = [a + b for a, b in zip(at, plan)]

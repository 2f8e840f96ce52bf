"""Small Birelix configurations and lively random weights for the tests.

The weights are not the package's random-model weights (N(0, 0.02) everywhere would leave every softmax flat, every gate at
one half and every decay alike): matrices are N(0, gain / sqrt(inputs)), the decays spread from a few tokens' memory to
hundreds, the convolutions' taps are all of a size, so that a wrong key, a window's edge that is one token off, a lost state
or tap, or a group of experts that was judged by one score moves the logits by far more than rounding does.  Everything is
rounded to bfloat16 before it is written, so that the engine in either precision and the plain implementation read the same
numbers.
"""
import json
import os

import numpy as np
import torch

import plain_birelix as P


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=2.0, groups=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=1000.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def attention(heads, kv_heads, dim, vdim, scale, window=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(vocab, width, layers, eps=1e-5, scale=None):
    cfg = {"architecture": "Birelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    return cfg


# sizes no fast kernel takes: a width that is no multiple of 16, heads of 9 to 20 channels, values of another size than keys,
# windows shorter than a page, three taps, experts of 10 and 20 inner channels, layers without a feed-forward, all experts chosen
ODD = config(97, 72, [
    delta(6, 2, 12, 20, 3, mlp=moe(5, 5, 20, 1.2)),
    latent(3, 10, 6, 14, 20, 18, 0.5, 300.0, mlp=dense(40)),
    attention(4, 2, 10, 12, 0.9, 7),
    delta(3, 3, 9, 5, 2, mlp=dense(24)),
    attention(3, 1, 20, 20, 0.7, 19, mlp=moe(4, 4, 10, 3.0, (2, 2))),
], scale=3.0)

# sizes the tensor-core kernels take (pages of 16): a latent layer with keys of 96 and values of 32 (keys and values raised by one
# product in portions) and one that folds, keys of 64 and 128 with values of 64, windows that end inside pages and one of
# exactly a page, delta heads of 32, 64 and 128 channels behind four taps
EVEN = config(160, 128, [
    latent(4, 64, 32, 32, 64, 48, 0.1, 10000.0, mlp=dense(96)),
    attention(4, 2, 64, 64, 0.2, 40, mlp=moe(3, 3, 32, 1.5)),
    delta(4, 2, 64, 64, 4, mlp=moe(4, 4, 48, 7.0, (2, 2))),
    attention(2, 1, 128, 64, 0.1, 16, mlp=dense(64)),
    delta(2, 2, 128, 32, 4),
    latent(3, 40, 16, 24, 56, 72, 0.15, 500.0, mlp=moe(2, 2, 64, 0.8)),
    delta(8, 4, 32, 128, 4, mlp=dense(48)),
])

# routers that choose: groups of two, three and one, kept singly and in pairs
ROUTED = config(120, 64, [
    delta(4, 2, 32, 16, 4, mlp=moe(8, 3, 24, 1.0, (4, 2))),
    attention(4, 4, 16, 16, 0.6, 33, mlp=moe(6, 2, 32, 2.5, (2, 1))),
    latent(2, 16, 8, 16, 24, 32, 0.5, 2000.0, mlp=moe(5, 2, 16, 1.5, (5, 3))),
], scale=1.5)

# what other configurations make larger: one head, one tap, a window of one position, one expert, narrow ranks and heads
ONES = config(50, 48, [
    delta(1, 1, 8, 5, 1, mlp=moe(1, 1, 8)),
    latent(1, 8, 2, 8, 4, 3, 0.5, 20.0, mlp=dense(16)),
    attention(1, 1, 16, 8, 0.5, 1),
    delta(2, 1, 3, 24, 4),
    attention(2, 2, 8, 16, 0.5),
])

# the delta rule alone (nothing is kept in pages): state columns beyond a block's, heads of more than 128 channels, seven taps
DELTAS = config(64, 40, [delta(2, 1, 130, 140, 7, mlp=dense(20)), delta(5, 5, 36, 8, 4), delta(4, 1, 200, 12, 5, mlp=moe(3, 3, 12))], scale=0.5)

CONFIGS = {"odd": ODD, "even": EVEN, "routed": ROUTED, "ones": ONES, "deltas": DELTAS}


def drawn_config(seed):
    """A configuration drawn from `seed`: two to six layers of any kind in any order, sizes from lists that hold what every kernel
    takes and what none does.  Routers send every token to all experts (a close call would decide for itself which way
    rounding goes)."""
    rng = np.random.default_rng(9000 + seed)
    pick = lambda xs: xs[int(rng.integers(0, len(xs)))]
    width = pick([64, 96, 136, 200, 256])

    def ff():
        r = rng.random()
        if r < 0.2:
            return None
        if r < 0.55:
            return dense(pick([32, 72, 128]))
        n, g = pick([(1, None), (2, None), (4, (2, 2)), (6, (3, 3))])
        return moe(n, n, pick([16, 24, 32, 20]), pick([0.7, 2.0, 7.0]), g)

    layers = []
    for _ in range(int(rng.integers(2, 7))):
        r = rng.random()
        if r < 0.3:
            D, R, V = pick([(64, 32, 32), (32, 32, 64), (24, 8, 40), (16, 16, 16), (48, 32, 80)])
            layers.append(latent(pick([1, 2, 5]), D, R, V, pick([32, 64, 100]), pick([24, 64, 90]), pick([1.0, 2.0]) / np.sqrt(D + R),
                                 pick([1e4, 1e6, 100.0]), ff()))
        elif r < 0.6:
            D, G = pick([16, 32, 64, 128, 40, 24, 96]), pick([1, 2, 3])
            Dv = pick([32, 64, 128]) if D in (64, 128) else pick([D, D, 20])
            layers.append(attention(G * pick([1, 2, 4]), G, D, Dv, pick([2.0, 3.0]) / np.sqrt(D), pick([None, 1, 15, 16, 48, 96, 200]), ff()))
        else:
            G = pick([1, 2, 3])
            layers.append(delta(G * pick([1, 2, 3]), G, pick([16, 32, 64, 128, 12, 72, 160]), pick([16, 32, 64, 9, 136]), pick([4, 4, 2, 3, 1, 6]), ff()))
    return config(pick([64, 300]), width, layers, scale=pick([None, 4.0]))


def tensor_shapes(cfg):
    E, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], E)
    for i, lay in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, lay["mixer"], lay.get("mlp")
        out[p + "norm1"] = (E,)
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        if lay["type"] == "latent_attention":
            R, C, r = m["rot_dim"], m["kv_rank"], m["q_rank"]
            out.update({p + "mix.dq": (r, E), p + "mix.dq.norm": (r,), p + "mix.uq": (H * (D + R), r), p + "mix.dkv": (C + R, E),
                        p + "mix.dkv.norm": (C,), p + "mix.uk": (H * D, C), p + "mix.uv": (H * Dv, C), p + "mix.g": (H, E)})
        elif lay["type"] == "attention":
            for x, rows in (("q", H * D), ("k", m["kv_heads"] * D), ("v", m["kv_heads"] * Dv)):
                out.update({p + "mix." + x: (rows, E), p + "mix." + x + ".b": (rows,)})
        else:
            for x, rows in (("q", m["kv_heads"] * D), ("k", m["kv_heads"] * D), ("v", H * Dv)):
                out.update({p + "mix." + x: (rows, E), p + "mix." + x + ".conv": (rows, m["conv"])})
            out.update({p + "mix.b": (H, E), p + "mix.a": (H, E), p + "mix.A_log": (H,), p + "mix.dt_bias": (H,), p + "mix.norm": (Dv,),
                        p + "mix.g": (H * Dv, E)})
        out[p + "mix.o"] = (E, H * Dv)
        if f is None:
            continue
        out[p + "norm2"] = (E,)
        groups = [""]
        if f["kind"] == "moe":
            out[p + "mlp.router"] = (f["router"]["experts"], E)
            groups = ["e%d." % e for e in range(f["router"]["experts"])]
        ff = f["ff"] if f["kind"] == "dense" else f["expert"]["ff"]
        for g in groups:
            out.update({p + "mlp." + g + "gate": (ff, E), p + "mlp." + g + "up": (ff, E), p + "mlp." + g + "down": (E, ff)})
    out["final.norm"] = (E,)
    return out


def lively_weights(cfg, seed):
    """{name: float64 array of bfloat16-representable values}."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if last == "A_log":
            x = rng.uniform(-4.0, 0.5, shape)          # exp(-exp(-4) softplus) forgets over a hundred tokens
        elif last == "dt_bias":
            x = rng.normal(-0.5, 1.0, shape)
        elif last == "conv":
            x = rng.normal(0.0, 0.7, shape)
        elif last == "b" and len(shape) == 1:
            x = rng.normal(0.0, 0.7, shape)            # biases of the projections
        elif len(shape) == 1:
            x = 1.0 + 0.2 * rng.normal(size=shape)     # norm weights
        elif name == "embed":
            x = rng.normal(0.0, 0.15 / (cfg.get("embedding") or {}).get("scale", 1.0), shape)
        else:
            gain = 2.0 if last in ("q", "k", "uq", "uk", "g", "a", "b", "router") else 1.0
            x = rng.normal(0.0, gain / np.sqrt(shape[1]), shape)
        w[name] = P.store_bfloat16(x)
    return w


def write_model(folder, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: torch.from_numpy(np.array(v, dtype=np.float64, order="C")).to(torch.bfloat16) for k, v in w.items()},
              os.path.join(folder, "model.safetensors"))
    return folder


def shifted_store(f):
    """Another realisation of the same rounding: the values are rounded a little beside themselves (x f rounded, then
    taken back, f near one), so every value falls elsewhere between its two neighbours; the error has the same size."""
    return lambda x: P.store_bfloat16(np.asarray(x) * f) / f


STORES = (P.store_bfloat16, shifted_store(1.0 + 2.0 ** -9), shifted_store(1.0 - 3.0 * 2.0 ** -10), shifted_store(1.0 + 5.0 * 2.0 ** -11))
CLOSE_CALL = 0.15   # of a router (see `plain_birelix.router_margins`); rounding to bfloat16 moves its logits by a few hundredths


class Oracle:
    """Exact logits [T, V] of one whole sequence and, per row, what rounding every stored activation to bfloat16 costs
    (root-mean-square distance from the exact row; the largest of four realisations of the rounding, since a softmax near a
    tie scatters a single one)."""

    def __init__(self, cfg, w, tokens, costs=True):
        self.exact = P.forward(cfg, w, tokens)
        self.cost = np.zeros(len(tokens))
        for store in STORES if costs else ():
            rounded = P.forward(cfg, w, tokens, store=store)
            self.cost = np.maximum(self.cost, np.sqrt(np.mean(np.square(rounded - self.exact), axis=1)))

    def __getitem__(self, row):
        return self.exact[row]


def decided_tokens(cfg, w, n, seed, tries=200):
    """Random tokens whose routers all decide clearly (a close call can go the other way under rounding and then reaches
    every later position through keys and state): each token is drawn until its own margins are wide, which later tokens
    do not change."""
    rng, toks = np.random.default_rng(seed), []
    while len(toks) < n:
        for _ in range(tries):
            toks.append(int(rng.integers(0, cfg["vocab"])))
            margins = []
            P.forward(cfg, w, toks, margins=margins)
            if min(m[-1] for m in margins) > CLOSE_CALL:
                break
            toks.pop()
        else:
            raise AssertionError("no token without a close call among %d tries" % tries)
    return toks


def compare(got, oracles_rows, dtype, what, judge):
    """`oracles_rows`: [(oracle, first row, one past the last)] in the order of `got`'s rows."""
    from helpers import assert_close
    want = np.concatenate([o.exact[a:b] for o, a, b in oracles_rows])
    cost = np.concatenate([o.cost[a:b] for o, a, b in oracles_rows])
    assert got.shape == want.shape and np.isfinite(got).all(), what
    assert_close(got, want, dtype, what, cost=cost, judge=judge)

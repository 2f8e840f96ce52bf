"""Small Negilorn configurations and lively random weights for the tests.

The weights are not the package's random-model weights (N(0, 0.02) everywhere would leave every softmax flat, every gate at
one half and every decay alike): matrices are N(0, gain / sqrt(inputs)), shares of the token shifts uniform in [0, 1), the
decays' offsets spread from a few tokens' memory to hundreds, so that a wrong key, a chunk's edge that is one token off, a
lost state, a row that was shifted by the wrong neighbour or a weight on the wrong side of an expert moves the logits by far
more than rounding does.  Everything is rounded to bfloat16 before it is written, so that the engine in either precision and
the plain implementation read the same numbers.
"""
import json
import os

import numpy as np
import torch

import plain_negilorn as N


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def attention(heads, kv_heads, dim, vdim, scale, rot=None, scaling=None, softcap=None, chunk=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if softcap:
        m["softcap"] = softcap
    if chunk:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def wkv(heads, dim, rank, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "rank": rank}, "mlp": mlp}


def config(vocab, width, layers, eps=1e-5, logit_scale=None):
    cfg = {"architecture": "Negilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if logit_scale is not None:
        cfg["logit_scale"] = logit_scale
    return cfg


# sizes no fast kernel takes: a width that is no multiple of 16, heads of 10, 12 and 20 channels, a rotation of a part of a
# head, values of another size than keys, chunks shorter than a page, a borrower whose chunks are longer than the owner's,
# experts of 10 and 20 inner channels, a middle width of 5, layers without a feed-forward, all experts chosen
ODD = config(97, 72, [
    attention(4, 2, 10, 12, 0.5, rot=(300.0, 6), scaling=(4.0, 1.0, 4.0, 16), softcap=5.0, chunk=7, mlp=dense(40)),
    wkv(3, 12, 5, mlp=moe(5, 5, 20, 12)),
    attention(4, 2, 10, 12, 0.6, rot=(300.0, 6), scaling=(4.0, 1.0, 4.0, 16), chunk=19, kv_from=0),
    wkv(2, 20, 9, mlp=dense(24)),
    attention(3, 3, 20, 20, 0.35, mlp=moe(4, 4, 10)),
], logit_scale=0.7)

# sizes the tensor-core kernels take (pages of 16): keys of 64 and 128 with values of 64, heads of 32 (equal sizes), chunks
# that end inside pages and one of exactly a page, two borrowers (one with its owner's chunks, one with shorter ones)
EVEN = config(160, 128, [
    attention(4, 2, 64, 64, 0.25, rot=(10000.0, 32), scaling=(2.0, 1.0, 4.0, 64), softcap=20.0, chunk=40, mlp=dense(96)),
    wkv(4, 32, 8, mlp=moe(3, 3, 32, 64)),
    attention(2, 1, 128, 64, 0.18, rot=(500.0, 128), softcap=9.0, chunk=50),
    wkv(2, 64, 24, mlp=dense(64)),
    attention(2, 1, 128, 64, 0.2, rot=(500.0, 128), chunk=50, kv_from=2, mlp=moe(2, 2, 48, 16)),
    attention(4, 2, 64, 64, 0.2, rot=(10000.0, 32), scaling=(2.0, 1.0, 4.0, 64), softcap=30.0, chunk=16, kv_from=0, mlp=dense(48)),
    attention(6, 2, 32, 32, 0.4, rot=(700.0, 32), chunk=96),
])

# routers that choose: more experts than a token uses, one of them by a single choice
ROUTED = config(120, 64, [
    wkv(2, 32, 6, mlp=moe(7, 2, 24, 40)),
    attention(4, 4, 16, 16, 0.5, rot=(1000.0, 16), softcap=12.0, chunk=33, mlp=moe(4, 1, 32, 8)),
    wkv(4, 16, 3, mlp=moe(6, 3, 16)),
], logit_scale=1.5)

# what other configurations make larger: one head, chunks of one position, one expert, a middle width of one, no chunks and no
# bound in the second attention
ONES = config(50, 48, [
    attention(1, 1, 16, 8, 0.5, rot=(20.0, 16), softcap=3.0, chunk=1, mlp=moe(1, 1, 8, 8)),
    wkv(1, 8, 1, mlp=dense(16)),
    attention(1, 1, 16, 8, 0.5, rot=(20.0, 2)),
    wkv(1, 24, 2),
])

# time mixing alone, no attention (nothing is kept in pages)
MIXING = config(64, 40, [wkv(5, 8, 4, mlp=dense(20)), wkv(2, 16, 12), wkv(1, 40, 7, mlp=moe(3, 3, 12, 20))], logit_scale=0.5)

CONFIGS = {"odd": ODD, "even": EVEN, "routed": ROUTED, "ones": ONES, "mixing": MIXING}


def drawn_config(seed):
    """A configuration drawn from `seed`: two to six layers of either kind in any order, sizes from lists that hold what every
    kernel takes and what none does, chunks of 1 to 200 positions or none, keys and values borrowed from any earlier owner.
    Routers send every token to all experts (a close call would decide for itself which way rounding goes)."""
    rng = np.random.default_rng(7000 + seed)
    pick = lambda xs: xs[int(rng.integers(0, len(xs)))]
    width = pick([64, 96, 136, 200, 256])

    def ff():
        r = rng.random()
        if r < 0.2:
            return None
        if r < 0.55:
            return dense(pick([32, 72, 128]))
        n = pick([1, 2, 4, 5])
        return moe(n, n, pick([16, 24, 32, 20]), pick([None, 32, 12]))

    owners = []

    def att(i):
        chunk = pick([None, 1, 15, 16, 48, 96, 200])
        softcap = pick([None, 4.0, 25.0])
        if owners and rng.random() < 0.4:
            j, m = owners[int(rng.integers(0, len(owners)))]
            lay = attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], pick([1.0, 2.0]) / np.sqrt(m["dim"]), None, None, softcap, chunk, j, ff())
            if "rot" in m:
                lay["mixer"]["rot"] = m["rot"]
            return lay
        D, G = pick([16, 32, 64, 128, 40, 24, 96]), pick([1, 2, 3])
        Dv = pick([32, 64, 128]) if D in (64, 128) else pick([D, D, 20])
        rot = None if rng.random() < 0.15 else (pick([1e4, 5e5, 100.0]), pick([D, D // 2 // 2 * 2]))
        scaling = None if rot is None or rng.random() < 0.4 else (pick([2.0, 8.0]), pick([1.0, 0.5]), pick([4.0, 2.0]), pick([32, 256, 2048]))
        lay = attention(G * pick([1, 2, 4]), G, D, Dv, pick([1.0, 2.0]) / np.sqrt(D), rot, scaling, softcap, chunk, None, ff())
        owners.append((i, lay["mixer"]))
        return lay

    layers = []
    for i in range(int(rng.integers(2, 7))):
        layers.append(att(i) if rng.random() < 0.5 else wkv(pick([1, 2, 3]), pick([16, 32, 64, 12, 72]), pick([4, 16, 33]), ff()))
    return config(pick([64, 300]), width, layers, logit_scale=pick([None, 0.5, 2.0]))


def tensor_shapes(cfg):
    E, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], E)
    for i, lay in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, lay["mixer"], lay.get("mlp")
        out.update({p + "norm1": (), p + "shift": (E,)})
        H, D = m["heads"], m["dim"]
        if lay["type"] == "attention":
            G, Dv = m["kv_heads"], m["vdim"]
            out.update({p + "mix.q": (H * D, E), p + "mix.g": (H, E), p + "mix.o": (E, H * Dv)})
            if m.get("kv_from") is None:
                out.update({p + "mix.k": (G * D, E), p + "mix.v": (G * Dv, E)})
        else:
            out.update({p + "mix.mu." + x: (E,) for x in "rkvgw"})
            out.update({p + "mix." + x: (H * D, E) for x in "rkvg"})
            out.update({p + "mix.o": (E, H * D), p + "mix.w1": (m["rank"], E), p + "mix.w2": (H * D, m["rank"]), p + "mix.w0": (H * D,),
                        p + "mix.u": (H, D), p + "mix.norm": (H * D,)})
        if f is None:
            continue
        out[p + "norm2"] = ()
        if f["kind"] == "dense":
            out.update({p + "mlp.gate": (f["ff"], E), p + "mlp.up": (f["ff"], E), p + "mlp.down": (E, f["ff"])})
        else:
            out[p + "mlp.router"] = (f["router"]["experts"], E)
            groups = [("e%d." % e, f["expert"]["ff"]) for e in range(f["router"]["experts"])]
            groups += [("shared.", f["shared"]["ff"])] if f.get("shared") else []
            for g, ff in groups:
                out.update({p + "mlp." + g + "up": (ff, E), p + "mlp." + g + "down": (E, ff)})
    out.update({"final.norm": (), "head": (cfg["vocab"], E)})
    return out


def lively_weights(cfg, seed):
    """{name: float64 array of bfloat16-representable values}."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if shape == ():
            x = np.array(1.0 + 0.2 * rng.normal())
        elif last == "shift" or ".mu." in name:
            x = rng.uniform(0.0, 1.0, shape)
        elif last == "w0":
            x = rng.normal(-2.0, 1.5, shape)           # exp(-exp(-2)) = 0.87; some channels remember hundreds of tokens
        elif last == "u":
            x = rng.normal(0.0, 1.0, shape)
        elif len(shape) == 1:
            x = 1.0 + 0.2 * rng.normal(size=shape)     # norm weights
        elif name == "embed":
            x = rng.normal(0.0, 1.0, shape)
        else:
            gain = 2.0 if last in ("q", "k", "g", "router") else 1.0
            x = rng.normal(0.0, gain / np.sqrt(shape[1]), shape)
        w[name] = N.store_bfloat16(x)
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
    return lambda x: N.store_bfloat16(np.asarray(x) * f) / f


STORES = (N.store_bfloat16, shifted_store(1.0 + 2.0 ** -9), shifted_store(1.0 - 3.0 * 2.0 ** -10), shifted_store(1.0 + 5.0 * 2.0 ** -11))
CLOSE_CALL = 0.1   # router logits spread over several units; rounding to bfloat16 moves them by a few hundredths


class Oracle:
    """Exact logits [T, V] of one whole sequence and, per row, what rounding every stored activation to bfloat16 costs
    (root-mean-square distance from the exact row; the largest of four realisations of the rounding, since a softmax near a
    tie scatters a single one).  `margin`: the smallest router margin of the sequence."""

    def __init__(self, cfg, w, tokens):
        margins, costs = [], []
        self.exact = N.forward(cfg, w, tokens, margins=margins)
        self.margin = float(np.min(margins)) if margins else np.inf
        for store in STORES:
            rounded = N.forward(cfg, w, tokens, store=store)
            costs.append(np.sqrt(np.mean(np.square(rounded - self.exact), axis=1)))
        self.cost = np.max(np.stack(costs), axis=0)

    def __getitem__(self, row):
        return self.exact[row]


def decided_tokens(cfg, w, n, seed, tries=60):
    """Random tokens whose routers all decide clearly (a close call can go the other way under rounding and then reaches
    every later position through keys and state): each token is drawn until its own margins are wide, which later tokens
    do not change."""
    rng, toks = np.random.default_rng(seed), []
    while len(toks) < n:
        for _ in range(tries):
            toks.append(int(rng.integers(0, cfg["vocab"])))
            margins = []
            N.forward(cfg, w, toks, margins=margins)
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

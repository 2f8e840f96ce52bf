"""Negilorn, plainly: numpy, float64, whole sequences, one function per mechanism.  It shares no code with the package and
knows no cache: every function takes all positions of one sequence at once.  `forward` takes the raw config.json
dictionary and a dictionary of arrays by tensor name.

Notation: the stream X [T, E]; h [T, E] what a sublayer reads, h[t] being position t; matrices are stored [out, in] and
applied as h W^T.  `store` (the identity by default) is applied to whatever an engine with 16-bit activations would keep
in them: the normed and shifted input, the outputs of matrix products, what feeds the next product.  With
`store_bfloat16` a run shows what such rounding costs; norms, angles, scores, softmax weights, decays, recurrent states,
router logits and the stream stay exact in either run.
"""
from __future__ import annotations

import math

import numpy as np


def store_bfloat16(x):
    """x rounded to bfloat16 (nearest even) and widened again."""
    a = np.ascontiguousarray(x, dtype=np.float32)
    bits = a.view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(x))


def same(x):
    return x


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_norm(x, g, eps):
    """RMS norm whose multiplier is one number."""
    return unit_rms(x, eps) * float(g)


def shifted(h):
    """Row t holds the row before it; row 0 holds zeros."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def token_shift(h, mu):
    """Channel c of h[t] moved the share mu[c] of the way to h[t - 1]."""
    return h + (shifted(h) - h) * mu


def rotary_frequencies(rot):
    """dims / 2 angular steps per position.  With `scaling` a channel pair of long wavelength (more than original / low
    positions) turns `factor` times slower, one of short wavelength (less than original / high) as before, and between
    the two the share of the old frequency grows linearly with original / wavelength."""
    dims, base = int(rot["dims"]), float(rot["base"])
    sc, out = rot.get("scaling"), []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wave, orig = 2.0 * math.pi / f, float(sc["original"])
            factor, low, high = float(sc["factor"]), float(sc["low"]), float(sc["high"])
            if wave > orig / low:
                f = f / factor
            elif wave >= orig / high:
                s = (orig / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return np.array(out)


def rotate_half(x, positions, rot):
    """x [T, heads, D]: channel i < dims/2 of every head is paired with channel i + dims/2 and the pair turned by
    position * frequency_i; channels from `dims` on pass."""
    dims = int(rot["dims"])
    half = dims // 2
    ang = np.asarray(positions, dtype=np.float64)[:, None] * rotary_frequencies(rot)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = np.array(x, dtype=np.float64)
    a, b = x[..., :half], x[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


def chunk_mask(T, size):
    """[T, T]: query i sees key j iff j <= i and both lie in the same run of `size` positions counted from 0 (0: one run)."""
    i = np.arange(T)
    seen = i[:, None] >= i[None, :]
    return seen & (i[:, None] // size == i[None, :] // size) if size else seen


def softmax_plus_one(scores, mask):
    """exp(s) / (1 + sum exp(s)) over the visible keys of each row."""
    s = np.where(mask, scores, -np.inf)
    top = np.maximum(s.max(axis=1, keepdims=True), 0.0)
    p = np.exp(s - top)
    return p / (np.exp(-top) + p.sum(axis=1, keepdims=True))


def bounded(scores, cap):
    return cap * np.tanh(scores / cap) if cap else scores


def attention_rows(h, P, m, positions, store=same):
    """What an attention layer with projections of its own keeps: rotated keys [T, G, D] and values [T, G, Dv]."""
    T, G = h.shape[0], m["kv_heads"]
    k = store(h @ P["k"].T).reshape(T, G, m["dim"])
    v = store(h @ P["v"].T).reshape(T, G, m["vdim"])
    if m.get("rot"):
        k = store(rotate_half(k, positions, m["rot"]))
    return k, v


def attention(h, P, m, positions, rows, store=same):
    """Queries of this layer over `rows` (k, v) of this layer or of the one it borrows them from."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k, v = rows
    q = store(h @ P["q"].T).reshape(T, H, D)
    if m.get("rot"):
        q = store(rotate_half(q, positions, m["rot"]))
    mask = chunk_mask(T, int((m.get("mask") or {}).get("size") or 0))
    gate = sigmoid(store(h @ P["g"].T))                     # [T, H]
    out = np.zeros((T, H, Dv))
    for n in range(H):
        g = n // (H // G)
        s = bounded((q[:, n] @ k[:, g].T) * m["scale"], float(m.get("softcap") or 0.0))
        out[:, n] = softmax_plus_one(s, mask) @ v[:, g] * gate[:, n:n + 1]
    return store(store(out.reshape(T, H * Dv)) @ P["o"].T)


def wkv_decay(mix_w, P, store=same):
    """exp(-exp(z)) per channel, z = W_w2 tanh(W_w1 mix_w) + w0."""
    return np.exp(-np.exp(np.tanh(mix_w @ P["w1"].T) @ P["w2"].T + P["w0"]))


def wkv_walk(r, k, v, w, u, state=None):
    """r, k, v, w [T, H, D], u [H, D]; S [H, D, D] rows are key channels.  o_t = (S + diag(u) k v^T)^T r, then
    S = diag(w) S + k v^T.  Returns (o [T, H, D], S)."""
    T, H, D = r.shape
    S = np.zeros((H, D, D)) if state is None else np.array(state, dtype=np.float64)
    o = np.zeros((T, H, D))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return o, S


def wkv(h, P, m, eps, store=same):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    mix = {x: store(token_shift(h, P["mu." + x])) for x in "rkvgw"}
    r, k, v = (store(mix[x] @ P[x].T).reshape(T, H, D) for x in "rkv")
    gate = silu(store(mix["g"] @ P["g"].T))
    w = wkv_decay(mix["w"], P, store).reshape(T, H, D)
    o, _ = wkv_walk(r, k, v, w, P["u"])
    y = unit_rms(o, eps).reshape(T, H * D) * P["norm"] * gate
    return store(store(y) @ P["o"].T)


def dense_feed_forward(h, P, store=same):
    return store(store(silu(h @ P["gate"].T) * (h @ P["up"].T)) @ P["down"].T)


def squared_relu(z):
    return np.square(np.maximum(z, 0.0))


def expert(h, up, down, store=same):
    return store(squared_relu(h @ up.T)) @ down.T


def route(h, W, top):
    """(chosen [T, top], weights [T, top]): the outputs of largest sigmoid score, lowest index first among equals."""
    s = sigmoid(h @ W.T)
    chosen = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def router_margins(h, W, top):
    """How far the last chosen logit lies above the first one left out, per token."""
    z = -np.sort(-(h @ W.T), axis=1)
    return np.full(len(z), np.inf) if top >= z.shape[1] else z[:, top - 1] - z[:, top]


def routed_feed_forward(h, P, m, store=same, margins=None):
    top = m["router"]["top"]
    chosen, weight = route(h, P["router"], top)
    if margins is not None:
        margins.append(router_margins(h, P["router"], top))
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weight[t]):
            y[t] += store(expert(w * h[t:t + 1], P["e%d.up" % e], P["e%d.down" % e], store))[0]
    if m.get("shared") is not None:
        y = y + store(expert(h, P["shared.up"], P["shared.down"], store))
    return store(y)


def sub(tensors, prefix):
    return {k[len(prefix):]: np.asarray(v, dtype=np.float64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens, store=same, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence.  `layers_out`, a list, receives the stream after every layer; `margins`, a list,
    the router margins [T] of every routed layer."""
    eps = float(config["norm"]["eps"])
    positions = np.arange(len(tokens))
    x = np.asarray(tensors["embed"], dtype=np.float64)[np.asarray(tokens)]
    kept = {}
    for i, layer in enumerate(config["layers"]):
        L = sub(tensors, "l%d." % i)
        P, m = sub(L, "mix."), layer["mixer"]
        h = store(token_shift(scalar_norm(x, L["norm1"], eps), L["shift"]))
        if layer["type"] == "wkv":
            # (the mixes are formed from the shifted input before it is rounded)
            y = wkv(token_shift(scalar_norm(x, L["norm1"], eps), L["shift"]), P, m, eps, store)
        else:
            j = m.get("kv_from")
            if j is None:
                kept[i] = attention_rows(h, P, m, positions, store)
            y = attention(h, P, m, positions, kept[i if j is None else j], store)
        x = x + y
        f = layer.get("mlp")
        if f is not None:
            h, F = store(scalar_norm(x, L["norm2"], eps)), sub(L, "mlp.")
            x = x + (dense_feed_forward(h, F, store) if f["kind"] == "dense" else routed_feed_forward(h, F, f, store, margins))
        if layers_out is not None:
            layers_out.append(x)
    x = store(scalar_norm(x, tensors["final.norm"], eps))
    return x @ np.asarray(tensors["head"], dtype=np.float64).T * float(config.get("logit_scale", 1.0))


def greedy_generate(config, tensors, prompt, n):
    """The n tokens that follow `prompt` when the most likely one is taken every time (the lowest index among equals)."""
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(np.argmax(forward(config, tensors, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out

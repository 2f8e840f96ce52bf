"""Birelix, plainly: numpy, float64, whole sequences, one function per mechanism.  It shares no code with the package and
knows no cache: every function takes all positions of one sequence at once.  `forward` takes the raw config.json
dictionary and a dictionary of arrays by tensor name.

Notation: the stream X [T, E]; h [T, E] what a sublayer reads, h[t] being position t; matrices are stored [out, in] and
applied as h W^T.  `store` (the identity by default) is applied to whatever an engine with 16-bit activations would keep
in them: the normed input, the outputs of matrix products, what feeds the next product.  With `store_bfloat16` a run shows
what such rounding costs; norms, angles, scores, softmax weights, unit vectors, decays, step sizes, recurrent states, router
logits and the stream stay exact in either run.
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


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def rotate_neighbours(x, positions, base):
    """x [T, heads, R]: channels (2i, 2i + 1) of every head are the pair turned by position * base^(-2i / R)."""
    R = x.shape[-1]
    f = np.array([base ** (-2.0 * i / R) for i in range(R // 2)])
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = np.empty(x.shape)
    u, v = x[..., 0::2], x[..., 1::2]
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def window_mask(T, size):
    """[T, T]: query i sees key j iff 0 <= i - j < size (size 0: every j <= i)."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < size) if size else d >= 0


def softmax(scores, mask, plus_one=False):
    """exp(s) / sum exp(s) over the visible keys of each row; with `plus_one` the denominator also holds one."""
    s = np.where(mask, scores, -np.inf)
    top = s.max(axis=1, keepdims=True)
    if plus_one:
        top = np.maximum(top, 0.0)
    p = np.exp(s - top)
    return p / (p.sum(axis=1, keepdims=True) + (np.exp(-top) if plus_one else 0.0))


def latent_attention(h, P, m, eps, positions, store=same):
    T, H, D, R, C, Dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["vdim"]
    base = float(m["rot"]["base"])
    cq = store(rms_norm(store(h @ P["dq"].T), P["dq.norm"], eps))
    q = store(cq @ P["uq"].T).reshape(T, H, D + R)
    down = store(h @ P["dkv"].T)
    c = store(rms_norm(down[:, :C], P["dkv.norm"], eps))
    r = store(rotate_neighbours(down[:, None, C:], positions, base))[:, 0]
    q_turned = store(rotate_neighbours(q[..., D:], positions, base))
    k, v = store(c @ P["uk"].T).reshape(T, H, D), store(c @ P["uv"].T).reshape(T, H, Dv)
    gate = sigmoid(store(h @ P["g"].T))                     # [T, H]
    mask, out = window_mask(T, 0), np.zeros((T, H, Dv))
    for n in range(H):
        s = (q[:, n, :D] @ k[:, n].T + q_turned[:, n] @ r.T) * m["scale"]
        out[:, n] = store(softmax(s, mask) @ v[:, n]) * gate[:, n:n + 1]
    return store(store(out.reshape(T, H * Dv)) @ P["o"].T)


def attention(h, P, m, eps, store=same):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = store(unit_rms(store(h @ P["q"].T + P["q.b"]).reshape(T, H, D), eps))
    k = store(unit_rms(store(h @ P["k"].T + P["k.b"]).reshape(T, G, D), eps))
    v = store(h @ P["v"].T + P["v.b"]).reshape(T, G, Dv)
    mask, out = window_mask(T, int((m.get("mask") or {}).get("size") or 0)), np.zeros((T, H, Dv))
    for n in range(H):
        g = n // (H // G)
        out[:, n] = softmax((q[:, n] @ k[:, g].T) * m["scale"], mask, plus_one=True) @ v[:, g]
    return store(store(out.reshape(T, H * Dv)) @ P["o"].T)


def short_convolution(x, w):
    """x [T, channels], w [channels, taps]: y[t] = sum_j w[:, taps - 1 - j] x[t - j], rows before the first being zero; then silu."""
    taps = w.shape[1]
    y = np.zeros_like(x)
    for j in range(min(taps, x.shape[0])):
        y[j:] += x[:x.shape[0] - j] * w[:, taps - 1 - j]
    return silu(y)


def unit_vector(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_walk(q, k, v, g, beta, state=None):
    """q, k [T, G, D], v [T, H, Dv], g, beta [T, H]; S [H, D, Dv].  S' = g S; u = beta (v - S'^T k); S = S' + k u^T; o = S^T q.
    Head h reads q and k of head h // (H / G).  Returns (o [T, H, Dv], S)."""
    T, G, D = q.shape
    H, Dv = v.shape[1:]
    head = np.arange(H) // (H // G)
    S = np.zeros((H, D, Dv)) if state is None else np.array(state, dtype=np.float64)
    o = np.zeros((T, H, Dv))
    for t in range(T):
        kt, qt = k[t, head], q[t, head]
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, qt)
    return o, S


def delta(h, P, m, eps, store=same):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (unit_vector(short_convolution(store(h @ P[x].T), P[x + ".conv"]).reshape(T, G, D)) for x in "qk")
    v = short_convolution(store(h @ P["v"].T), P["v.conv"]).reshape(T, H, Dv)
    beta = sigmoid(h @ P["b"].T)
    g = np.exp(-np.exp(P["A_log"]) * softplus(h @ P["a"].T + P["dt_bias"]))
    o, _ = delta_walk(q * D ** -0.5, k, v, g, beta)
    y = rms_norm(o, P["norm"], eps) * silu(store(h @ P["g"].T)).reshape(T, H, Dv)
    return store(store(y.reshape(T, H * Dv)) @ P["o"].T)


def dense_feed_forward(h, P, store=same):
    return store(store(gelu_tanh(h @ P["gate"].T) * (h @ P["up"].T)) @ P["down"].T)


def expert(h, gate, up, down, limit, store=same):
    g, u = np.minimum(h @ gate.T, limit), np.clip(h @ up.T, -limit, limit)
    return store(g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, W, router):
    """(chosen [T, top], weights [T, top]) by sigmoid scores: the `top` best outputs of the `keep` best groups, a group being
    judged by the sum of its two best scores; weights renormalised over the chosen."""
    s = sigmoid(h @ W.T)
    groups = router.get("groups") or {}
    n, keep = int(groups.get("count", 1)), int(groups.get("keep", 1))
    allowed = np.ones_like(s, dtype=bool)
    if keep < n:
        by_group = -np.sort(-s.reshape(len(s), n, -1), axis=2)
        best = np.argsort(-by_group[:, :, :2].sum(axis=2), axis=1, kind="stable")[:, :keep]
        allowed = np.zeros((len(s), n, s.shape[1] // n), dtype=bool)
        for t in range(len(s)):
            allowed[t, best[t]] = True
        allowed = allowed.reshape(s.shape)
    chosen = np.argsort(np.where(allowed, -s, np.inf), axis=1, kind="stable")[:, :router["top"]]
    w = np.take_along_axis(s, chosen, axis=1)
    return chosen, w / (w.sum(axis=1, keepdims=True) + 1e-20)


def router_margins(h, W, router):
    """How clearly each token's experts are chosen: the least change of one logit, about, that changes the choice.  The gap
    between the last expert chosen and the best one left out of the kept groups (in logits), and the gap between the last
    group kept and the best one left out (in scores, doubled: four logits move it, a score by at most a quarter of its logit)."""
    z = h @ W.T
    s = sigmoid(z)
    groups = router.get("groups") or {}
    n, keep, top = int(groups.get("count", 1)), int(groups.get("keep", 1)), router["top"]
    out = np.full(len(z), np.inf)
    for t in range(len(z)):
        zt = z[t].reshape(n, -1)
        score = np.array([np.sort(x)[::-1][:2].sum() for x in s[t].reshape(n, -1)])
        order = np.argsort(-score, kind="stable")
        if keep < n:
            out[t] = min(out[t], 2.0 * (score[order[keep - 1]] - score[order[keep]]))
        cand = np.sort(zt[order[:keep]].ravel())[::-1]
        if top < len(cand):
            out[t] = min(out[t], cand[top - 1] - cand[top])
    return out


def routed_feed_forward(h, P, m, store=same, margins=None):
    chosen, weight = route(h, P["router"], m["router"])
    if margins is not None:
        margins.append(router_margins(h, P["router"], m["router"]))
    limit, y = float(m["expert"]["limit"]), np.zeros_like(h)
    for e in range(P["router"].shape[0]):
        rows, which = np.nonzero(chosen == e)
        if len(rows):
            y[rows] += weight[rows, which][:, None] * store(expert(h[rows], P["e%d.gate" % e], P["e%d.up" % e], P["e%d.down" % e], limit, store))
    return store(y)


def sub(tensors, prefix):
    return {k[len(prefix):]: np.asarray(v, dtype=np.float64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens, store=same, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence.  `layers_out`, a list, receives the stream after every layer; `margins`, a list,
    the router margins [T] of every routed layer."""
    eps = float(config["norm"]["eps"])
    positions = np.arange(len(tokens))
    table = np.asarray(tensors["embed"], dtype=np.float64)
    x = table[np.asarray(tokens)] * float((config.get("embedding") or {}).get("scale", 1.0))
    for i, layer in enumerate(config["layers"]):
        L = sub(tensors, "l%d." % i)
        P, m = sub(L, "mix."), layer["mixer"]
        h = store(rms_norm(x, L["norm1"], eps))
        if layer["type"] == "latent_attention":
            y = latent_attention(h, P, m, eps, positions, store)
        elif layer["type"] == "attention":
            y = attention(h, P, m, eps, store)
        else:
            y = delta(h, P, m, eps, store)
        x = x + y
        f = layer.get("mlp")
        if f is not None:
            h, F = store(rms_norm(x, L["norm2"], eps)), sub(L, "mlp.")
            x = x + (dense_feed_forward(h, F, store) if f["kind"] == "dense" else routed_feed_forward(h, F, f, store, margins))
        if layers_out is not None:
            layers_out.append(x)
    return store(rms_norm(x, tensors["final.norm"], eps)) @ table.T


def greedy_generate(config, tensors, prompt, n):
    """The n tokens that follow `prompt` when the most likely one is taken every time (the lowest index among equals)."""
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(np.argmax(forward(config, tensors, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out

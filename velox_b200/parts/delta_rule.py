"""The gated delta rule: a recurrence whose state is corrected instead of added to.

    q, k = conv(W_q h), conv(W_k h)  [kv_heads, dim];  v = conv(W_v h)  [heads, vdim]
        (conv: a causal convolution over time, `conv_taps` taps per channel, zeros before the start, then silu)
    q, k per head as unit vectors x / sqrt(sum(x^2) + 1e-6), q times `q_scale`
    beta = sigmoid(W_b h),  g = exp(-exp(A_log) softplus(W_a h + dt_bias))    one number per head each
    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q              per head; head h reads q, k of head h / (heads / kv_heads)
    every head's o divided by its root mean square, times a weight [vdim], times silu(W_g h), projected by W_o

State per request, float32: S (transposed, [heads, vdim, dim]) and the convolutions' last inputs (a ring of `conv_taps` rows).
The projections of q, k, v and the gate are one matrix, those of a and b a second one whose sums stay float32; a decode step's
few rows take both in one product (`self.proj` holds all rows), with float32 sums.  A step of single tokens runs everything
between the projections in one kernel (`ops.delta_decode`); any other step runs convolution and recurrence
(`ops.delta_rule`, `csrc/delta_rule.cu`) and the norm per head with its gate.  Convolutions, unit vectors, decays, step sizes,
state, outputs, norm and gate are float32.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..csrc import ops
from .base import CacheParts, FixedState, Mixer, Runtime, TensorSpec
from .linear import Linear, matmul


class GatedDeltaRule(Mixer):
    cuda_graph_safe = True  # reads nothing of a step but device tensors and sizes fixed per graph
    KEYS = ("q", "k", "v", "g", "o", "b", "a", "A_log", "dt_bias", "norm")

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int,
                 conv_taps: int, eps: float = 1e-6, q_scale: Optional[float] = None, names: Sequence[str] = KEYS,
                 conv_suffix: str = ".conv"):
        super().__init__(prefix)
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.head_dim, self.v_head_dim, self.conv_taps, self.eps = int(head_dim), int(v_head_dim), int(conv_taps), float(eps)
        if min(self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim, self.conv_taps) <= 0 or self.num_heads % self.num_kv_heads:
            raise ValueError("%sdelta rule: sizes must be positive and the heads a multiple of the q/k heads" % prefix)
        for what, n, most in (("head_dim", self.head_dim, ops.DELTA_MAX_DIM), ("v_head_dim", self.v_head_dim, ops.DELTA_MAX_VDIM),
                              ("conv_taps", self.conv_taps, ops.DELTA_MAX_TAPS)):
            if n > most:
                raise ValueError("%s%s %d: the delta rule's kernels take up to %d" % (prefix, what, n, most))
        self.q_scale = self.head_dim ** -0.5 if q_scale is None else float(q_scale)
        self.names = dict(zip(self.KEYS, (prefix + n for n in names)))
        self.conv_names = [self.names[x] + conv_suffix for x in ("q", "k", "v")]
        self.proj = self.taps = self.neg_exp_a = self.dt_bias = self.norm_weight = None
        self.out: Optional[Linear] = None

    @property
    def channels(self) -> int:
        """What the convolutions run over: q, k, v."""
        return 2 * self.num_kv_heads * self.head_dim + self.num_heads * self.v_head_dim

    # -- weights -------------------------------------------------------------
    def tensor_specs(self) -> List[TensorSpec]:
        e, n, H = self.hidden_size, self.names, self.num_heads
        qk, vv, taps = self.num_kv_heads * self.head_dim, H * self.v_head_dim, self.conv_taps
        specs = [TensorSpec(n["q"], (qk, e), "matrix"), TensorSpec(n["k"], (qk, e), "matrix"), TensorSpec(n["v"], (vv, e), "matrix"),
                 TensorSpec(n["g"], (vv, e), "matrix"), TensorSpec(n["o"], (e, vv), "matrix"), TensorSpec(n["b"], (H, e), "matrix"),
                 TensorSpec(n["a"], (H, e), "matrix"), TensorSpec(n["A_log"], (H,), "bias"), TensorSpec(n["dt_bias"], (H,), "bias"),
                 TensorSpec(n["norm"], (self.v_head_dim,), "norm")]
        return specs + [TensorSpec(c, (rows, taps), "taps") for c, rows in zip(self.conv_names, (qk, qk, vv))]

    def bind(self, tensors: Dict[str, torch.Tensor], runtime: Runtime) -> None:
        super().bind(tensors, runtime)
        n, H = self.names, self.num_heads
        f32 = lambda t: t.to(torch.float32).contiguous()
        # rows: q, k, v, gate, (zeros up to a multiple of 8), b, a, (zeros likewise): every block starts on a 16-byte column
        wide = [tensors[n[x]] for x in ("q", "k", "v", "g")]
        self.g_col = self.channels
        self.ab_col = sum(w.shape[0] for w in wide)
        pad = lambda rows: [torch.zeros((rows, self.hidden_size), dtype=wide[0].dtype, device=wide[0].device)] if rows else []
        first = pad(-self.ab_col % 8)
        self.ab_col += sum(w.shape[0] for w in first)
        self.proj = torch.cat(wide + first + [tensors[n["b"]], tensors[n["a"]]] + pad(-2 * H % 8), dim=0).contiguous()
        self.taps = torch.cat([f32(tensors[c]) for c in self.conv_names], dim=0).t().contiguous()   # [taps, channels]
        self.neg_exp_a = -torch.exp(f32(tensors[n["A_log"]]))
        self.dt_bias, self.norm_weight = f32(tensors[n["dt_bias"]]), f32(tensors[n["norm"]])
        self.out = Linear(tensors[n["o"]])

    # -- state ---------------------------------------------------------------
    def cache_spec(self):
        return CacheParts((FixedState((self.conv_taps, self.channels), "float32"),
                           FixedState((self.num_heads, self.v_head_dim, self.head_dim), "float32")))

    # -- step ----------------------------------------------------------------
    def forward(self, h: torch.Tensor, ctx, cache) -> torch.Tensor:
        G, D, H, Dv = self.num_kv_heads, self.head_dim, self.num_heads, self.v_head_dim
        ring, state = (part.state for part in cache.parts)
        if h.dtype == torch.float32 or ops.skinny_supported(h.shape[0], self.hidden_size, h, self.proj):
            x = matmul(h, self.proj, None, torch.float32)   # [tokens, q | k | v | g | b | a]: float32 sums
            ab = x[:, self.ab_col:]
        else:
            x = matmul(h, self.proj[:self.ab_col])
            ab = matmul(h, self.proj[self.ab_col:], None, torch.float32)
        more = (self.taps, self.neg_exp_a, self.dt_bias)
        if ctx.decode_only:
            y = ops.delta_decode(x, self.g_col, ab, H, 0, *more, self.norm_weight, state, ring, ctx, G, D, H, Dv, self.q_scale,
                                 self.eps, h.dtype)
        else:
            o = ops.delta_rule(x, ab, H, 0, *more, state, ring, ctx, G, D, H, Dv, self.q_scale)
            y = ops.head_norm_gate(o, x[:, self.g_col:self.g_col + H * Dv], self.norm_weight, H, self.eps, "silu", out_dtype=h.dtype)
        return self.out(y)

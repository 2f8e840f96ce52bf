"""RWKV-style time mixing: a recurrence whose decay follows the input, channel by channel, and whose current token enters
the output with a weight of its own.

Every projection reads its own mix of the token and the one before it, m_x = h + (h' - h) mu_x for x in r, k, v, g, w
(h' of a request's first token is zero):
    r, k, v = W_r m_r, W_k m_k, W_v m_v  per head;  gate = silu(W_g m_g);  log a = -exp(W_w2 tanh(W_w1 m_w) + w0)
    o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t;  S_t = diag(a_t) S_(t-1) + k_t v_t^T
Each head's o is divided by its root mean square; the heads are joined, times `norm`, times the gate, and projected by W_o.

State per request, float32: the last h [hidden] and S [heads, dim, dim].  The recurrence is `ops.linear_attention_walk` with a
bonus (`csrc/state_mixers.cu`); decays are float32 from the narrow projection's sums on (`ops.low_rank_decay`).  A block that
norms and shifts the stream can make the five mixes in its own kernel and call `forward_mixed`; `forward` makes them itself.
The five input projections are one matrix here ([W_r; W_k; W_v; W_g; W_w1]): a decode step streams it in one launch, each
row block with its own input (`ops.gemm_inputs`, float32 sums); larger steps run the first four as a batch of products.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..csrc import ops
from .base import CacheParts, FixedState, Mixer, Runtime, TensorSpec
from .linear import Linear, matmul
from .linear_attention import step_stretches


class WkvMixer(Mixer):
    cuda_graph_safe = True  # reads nothing of a step but device tensors and sizes fixed per graph
    MIXES = ("r", "k", "v", "g", "w")
    KEYS = ("r", "k", "v", "g", "o", "w1", "w2", "w0", "u", "norm")

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, head_dim: int, eps: float = 1e-6,
                 decay_rank: Optional[int] = None, names: Sequence[str] = KEYS, mix_prefix: str = "mu."):
        super().__init__(prefix)
        self.hidden_size, self.num_heads, self.head_dim, self.eps = int(hidden_size), int(num_heads), int(head_dim), float(eps)
        if not 0 < self.head_dim <= ops.LINEAR_ATTENTION_MAX_DIM:
            raise ValueError("%shead_dim %d: the recurrence kernel takes up to %d" % (prefix, head_dim, ops.LINEAR_ATTENTION_MAX_DIM))
        # rows of W_w1; None: read off the tensor when it is bound
        self.decay_rank: Optional[int] = int(decay_rank) if decay_rank else None
        self.names = dict(zip(self.KEYS, (prefix + n for n in names)))
        self.mix_names = [prefix + mix_prefix + x for x in self.MIXES]
        self.mixes = self.proj = self.decay_up = self.decay_bias = self.bonus = self.norm_weight = None
        self.out: Optional[Linear] = None

    # -- weights -------------------------------------------------------------
    def tensor_specs(self) -> List[TensorSpec]:
        e, hd, n = self.hidden_size, self.num_heads * self.head_dim, self.names
        r = self.decay_rank or -1   # (not given: whatever the file holds)
        specs = [TensorSpec(m, (e,), "share") for m in self.mix_names]
        specs += [TensorSpec(n[x], (hd, e), "matrix") for x in ("r", "k", "v", "g")]
        return specs + [TensorSpec(n["o"], (e, hd), "matrix"), TensorSpec(n["w1"], (r, e), "matrix"),
                        TensorSpec(n["w2"], (hd, r), "matrix_f32"), TensorSpec(n["w0"], (hd,), "bias"),
                        TensorSpec(n["u"], (self.num_heads, self.head_dim), "bias"), TensorSpec(n["norm"], (hd,), "norm")]

    def bind(self, tensors: Dict[str, torch.Tensor], runtime: Runtime) -> None:
        super().bind(tensors, runtime)
        n = self.names
        f32 = lambda t: t.to(torch.float32).contiguous()
        self.mixes = torch.stack([f32(tensors[m]) for m in self.mix_names]).contiguous()
        self.proj = torch.cat([tensors[n[x]] for x in ("r", "k", "v", "g", "w1")], dim=0).contiguous()
        up = f32(tensors[n["w2"]])
        self.decay_rank = int(up.shape[1])
        if self.proj.shape[0] != 4 * self.num_heads * self.head_dim + self.decay_rank:
            raise ValueError("%s and %s disagree about the middle width of the decay's projection" % (n["w1"], n["w2"]))
        if self.decay_rank > ops.LOW_RANK_DECAY_MAX_RANK:
            raise ValueError("%s: the decay kernel takes a middle width of up to %d, got %d"
                             % (n["w2"], ops.LOW_RANK_DECAY_MAX_RANK, self.decay_rank))
        self.decay_up = up.t().contiguous()   # [rank, channels]: the kernel's threads read neighbouring channels
        self.decay_bias, self.bonus, self.norm_weight = f32(tensors[n["w0"]]), f32(tensors[n["u"]]), f32(tensors[n["norm"]])
        self.out = Linear(tensors[n["o"]])

    # -- state -----------------------------------------------------------------
    def cache_spec(self):
        return CacheParts((FixedState((self.hidden_size,), "float32"),
                           FixedState((self.num_heads, self.head_dim, self.head_dim), "float32")))

    def mix_state(self, cache) -> torch.Tensor:
        """Where the last h of every request lies: float32 [slots, hidden]."""
        return cache.parts[0].state

    # -- step ------------------------------------------------------------------
    def forward(self, h: torch.Tensor, ctx, cache) -> torch.Tensor:
        return self.forward_mixed(ops.shift_mix(h, self.mixes, ctx, self.mix_state(cache)), ctx, cache)

    def forward_mixed(self, mixed: torch.Tensor, ctx, cache) -> torch.Tensor:
        """`mixed` [5, tokens, hidden]: the mixes that r, k, v, g and the decay read."""
        H, D = self.num_heads, self.head_dim
        HD, tokens = H * D, mixed.shape[1]
        if mixed.dtype == torch.bfloat16 and ops.skinny_supported(tokens, self.hidden_size, mixed[0], self.proj):
            x = ops.gemm_inputs(mixed, self.proj, HD, torch.float32)   # [tokens, r | k | v | g | w1]
            low, gate, cols = x[:, 4 * HD:], x[:, 3 * HD:4 * HD], (0, HD, 2 * HD)
        else:
            x = ops.gemm_members(mixed[:4], self.proj[:4 * HD].view(4, HD, self.hidden_size))   # [r, k, v, g][tokens, H D]
            low, gate, cols = matmul(mixed[4], self.proj[4 * HD:], None, torch.float32), x[3], (0, tokens * HD, 2 * tokens * HD)
        log_decay = ops.low_rank_decay(low, self.decay_up, self.decay_bias)
        o = ops.linear_attention_walk(x, *cols, cache.parts[1].state, ctx.cu_seqlens, ctx.state_slots, ctx.n_seqs, H, D, D,
                                      gate=log_decay, gate_is_log=True, bonus=self.bonus, stretches=step_stretches(ctx))
        return self.out(ops.head_norm_gate(o, gate, self.norm_weight, H, self.eps, "silu", out_dtype=mixed.dtype))

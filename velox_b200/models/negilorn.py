"""Negilorn as a plan of parts.

Input: the token's row.  Every layer is the pre-norm layer whose mixer reads a shifted input (`token_shift`); norms are RMS
norms with one number as their multiplier.  The mixer is, layer by layer as config.json lists them, one of
  * softmax attention over a paged cache: grouped key/value heads, values of a size of their own, q and k rotated on their
    first channels with halves paired (the frequencies optionally stretched by wavelength), a score multiplier and a tanh
    bound on the scores, a mask that cuts the sequence into chunks, one added to the softmax's denominator, a sigmoid gate
    per head.  A layer may read the keys and values that an earlier layer cached instead of making its own;
  * RWKV-style time mixing (`wkv`).
The feed-forward is gated with silu, or routed (experts down(relu(up(w h))^2) chosen by sigmoid scores whose weight w
multiplies the expert's input, plus a shared expert of the same form), or absent.  Output: norm, head, logits times a number.
Tensor names: `l<i>.` plus `norm1 | norm2 | shift | mix.{q,k,v,g,o} | mix.{mu.r,mu.k,mu.v,mu.g,mu.w,r,k,v,g,o,w1,w2,w0,u,norm}
| mlp.{gate,up,down} | mlp.{router,e<n>.up,e<n>.down,shared.up,shared.down}`, `embed`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.model_config import NegilornConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec

# fixed by the design: the experts' activation, the dense feed-forward's, the score of the entry without a value
EXPERT_ACTIVATION = "relu2"
DENSE_ACTIVATION = "silu"
SINK_SCORE = 0.0


def _mixer(cfg: NegilornConfig, i: int, p: str) -> PartSpec:
    layer = cfg.layers[i]
    m = layer["mixer"]
    if layer["type"] == "wkv":
        return PartSpec("wkv", p, dict(hidden_size=cfg.width, num_heads=m["heads"], head_dim=m["dim"], eps=cfg.norm_eps,
                                       decay_rank=m.get("rank")))
    rot, position = m.get("rot"), None
    if rot:
        position = PartSpec("rotary", "", dict(head_dim=m["dim"], theta=float(rot["base"]), rotary_dim=int(rot.get("dims") or m["dim"]),
                                               layout="half", scaling=rot.get("scaling")))
    return PartSpec("paged_attention", p, dict(
        hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"], bias=False,
        qk_norm=False, eps=cfg.norm_eps, scale=float(m["scale"]), score_softcap=float(m.get("softcap") or 0.0), position=position,
        names=("q", "k", "v", "o"), output_gate=True, gate_name="g", sink_value=SINK_SCORE, weights_32bit=True,
        chunk=cfg.chunk_of(i), own_kv=cfg.kv_source(i) is None,
        reader_chunks=[cfg.chunk_of(j) for j in range(len(cfg.layers)) if cfg.kv_source(j) == i]))


def _feed_forward(cfg: NegilornConfig, mlp, p: str):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("gated_mlp", p, dict(hidden_size=cfg.width, intermediate_size=mlp["ff"], activation=DENSE_ACTIVATION,
                                             names=("gate", "up", "down")))
    shared = None
    if mlp.get("shared") is not None:
        shared = PartSpec("dense_mlp", p + "shared.", dict(hidden_size=cfg.width, intermediate_size=mlp["shared"]["ff"],
                                                           activation=EXPERT_ACTIVATION, names=("up", "down")))
    return PartSpec("routed_experts", p, dict(
        hidden_size=cfg.width, experts=mlp["router"]["experts"], top=mlp["router"]["top"], intermediate_size=mlp["expert"]["ff"],
        activation=EXPERT_ACTIVATION, router_bias=False, shared=shared, names=("up", "down"), scores="sigmoid", gated=False,
        weight_input=True))


def negilorn_plan(cfg: NegilornConfig) -> ModelPlan:
    norm = lambda name: PartSpec("rms_norm", name, dict(size=cfg.width, eps=cfg.norm_eps, weight_name="", scalar=True))
    layers, unused = [], []
    for i, layer in enumerate(cfg.layers):
        p = "l%d." % i
        ff = _feed_forward(cfg, layer.get("mlp"), p + "mlp.")
        norms = {"mixer": norm(p + "norm1")}
        if ff is not None:
            norms["feed_forward"] = norm(p + "norm2")
        else:   # (a layer without a feed-forward has no use for its norm, should a checkpoint carry it)
            unused.append(p + "norm2")
        layers.append(LayerSpec(mixer=_mixer(cfg, i, p + "mix."), feed_forward=ff, norms=norms, block="token_shift",
                                cache_of=cfg.kv_source(i), block_params=dict(hidden_size=cfg.width, shift_name=p + "shift")))
    return ModelPlan(
        vocab_size=cfg.vocab, hidden_size=cfg.width,
        embedding=PartSpec("token_embedding", "", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, weight_name="embed")),
        layers=layers, final_norm=norm("final.norm"),
        head=PartSpec("linear_head", "head", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, weight_name="",
                                                  logit_scale=cfg.logit_scale)),
        ignored_tensors=unused)


register_architecture(NegilornConfig.architecture, NegilornConfig.model_type, NegilornConfig, negilorn_plan)

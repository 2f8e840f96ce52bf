"""Birelix as a plan of parts.

Input: the token's row times a multiplier.  Every layer is the pre-norm layer (RMS norms with a weight per channel).  The mixer
is, layer by layer as config.json lists them, one of
  * latent attention: queries through a normed latent vector of their own, keys and values raised from one normed latent vector
    per position plus a rotated key part that the heads share (neighbours paired), a sigmoid gate per head;
  * softmax attention without rotation: grouped key/value heads, values of a size of their own, biases on q, k and v, q and k
    divided by their root mean square per head, a sliding window, one added to the softmax's denominator;
  * the gated delta rule behind short convolutions (`gated_delta_rule`).
The feed-forward is gated with the tanh form of gelu, or routed, or absent: experts with a bounded gate, chosen by sigmoid scores
inside the best groups of neighbours (a group is judged by its two best scores) and weighted by the scores divided by their sum.
Output: norm, then the embedding table itself as the head.
Tensor names: `l<i>.` plus `norm1 | norm2 | mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,g,o} | mix.{q,q.b,k,k.b,v,v.b,o}
| mix.{q,q.conv,k,k.conv,v,v.conv,b,a,A_log,dt_bias,norm,g,o} | mlp.{gate,up,down} | mlp.{router,e<n>.gate,e<n>.up,e<n>.down}`,
`embed`, `final.norm`.
"""
from __future__ import annotations

from ..config.model_config import BirelixConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec

# fixed by the design: the dense feed-forward's activation, the slope of the experts' gate, the score of the entry without a value
DENSE_ACTIVATION = "gelu_pytorch_tanh"
EXPERT_SLOPE = 1.702
SINK_SCORE = 0.0


def _mixer(cfg: BirelixConfig, layer: dict, p: str) -> PartSpec:
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return PartSpec("latent_attention", p, dict(
            hidden_size=cfg.width, num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"],
            kv_rank=m["kv_rank"], scale=float(m["scale"]), eps=cfg.norm_eps, q_rank=m["q_rank"], head_gate=True,
            position=PartSpec("rotary", "", dict(head_dim=m["rot_dim"], theta=float(m["rot"]["base"]), rotary_dim=m["rot_dim"],
                                                 layout="interleaved"))))
    if layer["type"] == "attention":
        return PartSpec("paged_attention", p, dict(
            hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
            bias=True, bias_suffix=".b", out_bias=False, qk_norm=True, qk_norm_weight=False, eps=cfg.norm_eps,
            window=cfg.window_of(m), scale=float(m["scale"]), position=None, names=("q", "k", "v", "o"), sink_value=SINK_SCORE,
            weights_32bit=True))
    return PartSpec("gated_delta_rule", p, dict(
        hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
        conv_taps=m["conv"], eps=cfg.norm_eps))


def _feed_forward(cfg: BirelixConfig, mlp, p: str):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("gated_mlp", p, dict(hidden_size=cfg.width, intermediate_size=mlp["ff"], activation=DENSE_ACTIVATION,
                                             names=("gate", "up", "down")))
    router = mlp["router"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    return PartSpec("routed_experts", p, dict(
        hidden_size=cfg.width, experts=router["experts"], top=router["top"], intermediate_size=mlp["expert"]["ff"],
        router_bias=False, names=("gate", "up", "down"), scores="sigmoid", groups=groups["count"], keep_groups=groups["keep"],
        group_pair=True, renormalise=True, capped=(float(mlp["expert"]["limit"]), EXPERT_SLOPE)))


def birelix_plan(cfg: BirelixConfig) -> ModelPlan:
    norm = lambda name: PartSpec("rms_norm", name, dict(size=cfg.width, eps=cfg.norm_eps, weight_name=""))
    layers, unused = [], []
    for i, layer in enumerate(cfg.layers):
        p = "l%d." % i
        ff = _feed_forward(cfg, layer.get("mlp"), p + "mlp.")
        norms = {"mixer": norm(p + "norm1")}
        if ff is not None:
            norms["feed_forward"] = norm(p + "norm2")
        else:   # (a layer without a feed-forward has no use for its norm, should a checkpoint carry it)
            unused.append(p + "norm2")
        layers.append(LayerSpec(mixer=_mixer(cfg, layer, p + "mix."), feed_forward=ff, norms=norms, block="pre_norm"))
    return ModelPlan(
        vocab_size=cfg.vocab, hidden_size=cfg.width,
        embedding=PartSpec("token_embedding", "", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, weight_name="embed",
                                                       scale=cfg.embedding_scale)),
        layers=layers, final_norm=norm("final.norm"),
        head=PartSpec("linear_head", "head", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, weight_name="", tied=True)),
        ignored_tensors=unused)


register_architecture(BirelixConfig.architecture, BirelixConfig.model_type, BirelixConfig, birelix_plan)

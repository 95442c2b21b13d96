"""Kuvelix on the B200 engine: a layer-list decoder of parallel attention / feed-forward blocks with experts that may do nothing.

`config.json`: `architecture: "Kuvelix"`, `width`, `vocab`, `norm.eps`, `loop` and `layers`. The token embedding passes a weighted RMS
norm; a layer is `x += mixer(u) + ff(u)` with ONE weighted RMS norm `u = rms_w(x)` that both sublayers read; `loop: {start, stop,
times}` runs a block of layers several times in a row with the same tensors, every pass on a cache of its own and with nothing added
between the passes; the head is the embedding table behind a final norm. Mixer: `attention` (grouped heads; biases on q, k and v;
weighted RMS norm of every q and k head; rotary pairs of neighbours on the leading dimensions, all frequencies divided by one factor
when the rotation is scaled; causal softmax; a sigmoid output gate per channel). Feed-forwards: `dense`, `W_down (gelu(W_gate h) *
(W_up h))` with the tanh form of GELU, and `moe`, bounded gated experts `W_down (a(g) (u + 1))` with `g = min(W_gate h, limit)`,
`u = clamp(W_up h, +-limit)`, `a(g) = g sigmoid(1.702 g)` behind a softmax router: scores plus a learned correction choose the groups
(by their best member) and the experts, the scores alone, over their sum, are the weights, and the last `identity` rows of the router
are identity experts, whose output is `h`. This module only reads the configuration; tensors, engine, generation and replay are the
layer-list decoders' common code (layer_list.py).
"""
from ..._b2 import (BLOCK_PARALLEL_RMS, FF_GELU_GLU, FF_MOE, GATE_CHANNEL, MASK_CAUSAL, MIXER_GQA_ATTN, MOE_ACT_CLAMP_GLU, MOE_GROUP_MAX,
                    MOE_SCORE_SOFTMAX, QK_NORM_HEAD, ROT_LINEAR)
from .layer_list import LayerListConfig, LayerListForCausalLM

EXPERT_SLOPE = 1.702   # a(g) = g sigmoid(1.702 g): the sigmoid approximation of GELU, fixed by the design


def _rotation(rot, what):
    """Engine fields of a `rot` entry (absent: no rotation): rotated dimensions, base and, when present, the linear scaling."""
    if not rot or not int(rot.get("dims", 0)):
        return dict(rot_dims=0, rot_base=10000.0)
    d = dict(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]))
    sc = rot.get("scaling")
    if sc:
        if float(sc["factor"]) <= 0:
            raise ValueError(f"{what}: rot.scaling.factor must be positive")
        d.update(rot_scaling=ROT_LINEAR, rot_factor=float(sc["factor"]))
    return d


def _experts(mlp):
    """Engine fields of a mixture of experts; absent groups are one group, absent identity experts none, an absent limit no bound."""
    r, ex = mlp["router"], mlp["expert"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return dict(ff_kind=FF_MOE, ff=int(ex["ff"]), moe_act=MOE_ACT_CLAMP_GLU, ff_limit=float(ex.get("limit") or 0.0), ff_act_slope=EXPERT_SLOPE,
                moe_experts=int(r["experts"]), moe_identity=int(r.get("identity") or 0), moe_top=int(r["top"]), moe_groups=int(groups["count"]),
                moe_keep=int(groups["keep"]), moe_score=MOE_SCORE_SOFTMAX, moe_group_score=MOE_GROUP_MAX, moe_scale=1.0, moe_correction=1)


class KuvelixConfig(LayerListConfig):
    model_type = "Kuvelix"

    def model_desc(self):
        d = dict(block=BLOCK_PARALLEL_RMS, residual_mult=1.0, embed_norm=1, tied_head=1)
        loop = self.raw.get("loop")
        if loop:
            d.update(loop_start=int(loop["start"]), loop_stop=int(loop["stop"]), loop_times=int(loop["times"]), loop_plain=1)
        return d

    def layer_descs(self, shapes):
        out = []
        for i, layer in enumerate(self.layers):
            mix, mlp, kind = layer["mixer"], layer.get("mlp"), layer["type"]
            if kind != "attention":
                raise NotImplementedError(f"layer {i}: mixer type {kind!r}")
            d = dict(weights_of=-1, ff=0, type=MIXER_GQA_ATTN, ga_heads=int(mix["heads"]), ga_kv_heads=int(mix.get("kv_heads", mix["heads"])),
                     ga_dim=int(mix["dim"]), ga_vdim=int(mix.get("vdim", mix["dim"])), ga_scale=float(mix["scale"]), ga_qkv_bias=1, ga_qk_norm=QK_NORM_HEAD,
                     ga_gate=GATE_CHANNEL, mask_kind=MASK_CAUSAL, **_rotation(mix.get("rot"), f"layer {i}"))
            if mlp:
                ff_kind = mlp.get("kind", "dense")
                if ff_kind == "dense":
                    d.update(ff_kind=FF_GELU_GLU, ff=int(mlp["ff"]))
                elif ff_kind == "moe":
                    d.update(_experts(mlp))
                else:
                    raise NotImplementedError(f"layer {i}: feed-forward kind {ff_kind!r}")
            out.append(d)
        return out


class KuvelixForCausalLM(LayerListForCausalLM):
    """Holds the checkpoint tensors (CPU) and builds the device engine on first use.

    dtype: torch.bfloat16 = bf16 matrix products with fp32 accumulation on bf16 weights (norms, rotations, scores and softmax, router,
    gates, the caches and the residual stream in fp32); torch.float32 = everything in true fp32."""
    config_class = KuvelixConfig

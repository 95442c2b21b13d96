"""Ramosun on the B200 engine: a layer-list decoder of parallel blocks whose norms compute no statistics.

`config.json`: `architecture: "Ramosun"`, `width`, `vocab`, `norm.eps`, `logit_softcap`, `loop` and `layers`. A layer is
`x += mixer(N1(x)) + ff(N2(x))`, both norms of the same x, with the dynamic tanh `N(x) = tanh(alpha x) w + b`; `loop: {start, stop,
times}` runs a block of layers several times in a row with the same tensors, every pass on a cache / state of its own, and x becomes
`W_in [x; x0]` (x0: the embedding output) in front of every pass. Mixers: `mlstm` (matrix memory per head with exponential input and
forget gates, kept in range by a running maximum, its normaliser beside it; per-head RMS norm, sigmoid gate), `delta` (gated delta
rule: unit q and k behind a short convolution with SiLU, one decay and one write strength per head; per-head RMS norm, SiLU gate) and
`attention` (grouped heads whose values are the raw keys, a weighted RMS norm over the whole query and the whole key projection,
rotate-half positions with frequencies scaled by bands of wavelength, a sliding window, a learned sink per head). Feed-forward:
`W_down gelu(W_up h)`, the erf form. The head is the embedding table; logits are soft-capped. This module only reads the
configuration; tensors, engine, generation and replay are the layer-list decoders' common code (layer_list.py).
"""
from ..._b2 import (BLOCK_PARALLEL2, FF_GELU, GATE_NONE, MASK_CAUSAL, MASK_WINDOW, MIXER_DELTA, MIXER_GQA_ATTN, MIXER_MLSTM, NORM_DYT, QK_NORM_ALL,
                    ROT_BANDS, SINK_HEAD)
from .layer_list import LayerListConfig, LayerListForCausalLM


def _rotation(rot, what):
    """Engine fields of a `rot` entry (absent: no rotation): rotated dimensions, base and, when present, the scaling by bands."""
    if not rot or not int(rot.get("dims", 0)):
        return dict(rot_dims=0, rot_base=10000.0)
    d = dict(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]))
    sc = rot.get("scaling")
    if sc:
        if float(sc["factor"]) <= 0:
            raise ValueError(f"{what}: rot.scaling.factor must be positive")
        d.update(rot_scaling=ROT_BANDS, rot_factor=float(sc["factor"]), rot_original=float(sc["original"]), rot_fast=float(sc["high"]),
                 rot_slow=float(sc["low"]))
    return d


class RamosunConfig(LayerListConfig):
    model_type = "Ramosun"

    def model_desc(self):
        c = self.raw
        d = dict(block=BLOCK_PARALLEL2, norm_kind=NORM_DYT, residual_mult=1.0, tied_head=1, logit_softcap=float(c.get("logit_softcap") or 0.0))
        loop = c.get("loop")
        if loop:
            d.update(loop_start=int(loop["start"]), loop_stop=int(loop["stop"]), loop_times=int(loop["times"]), loop_mix=1)
        return d

    def layer_descs(self, shapes):
        out = []
        for i, layer in enumerate(self.layers):
            mix, mlp, kind = layer["mixer"], layer.get("mlp"), layer["type"]
            d = dict(weights_of=-1, ff=0)
            heads, dim = int(mix["heads"]), int(mix["dim"])
            if kind == "mlstm":
                d.update(type=MIXER_MLSTM, ml_heads=heads, ml_dim=dim, ml_vdim=int(mix["vdim"]), ml_cap=float(mix["gate_cap"]))
            elif kind == "delta":
                taps = mix.get("conv")
                if taps is None:      # what the checkpoint's tensor says when the configuration is silent
                    taps = shapes[f"l{i}.mix.q.conv"][1]
                d.update(type=MIXER_DELTA, dn_heads=heads, dn_kv_heads=int(mix.get("kv_heads", heads)), dn_dim=dim, dn_vdim=int(mix["vdim"]),
                         dn_conv=int(taps))
            elif kind == "attention":
                if int(mix.get("vdim", dim)) != dim:
                    raise ValueError(f"layer {i}: the values are the keys, so vdim must equal dim")
                size = (mix.get("mask") or {}).get("size")
                d.update(type=MIXER_GQA_ATTN, ga_heads=heads, ga_kv_heads=int(mix.get("kv_heads", heads)), ga_dim=dim, ga_vdim=dim, ga_key_values=1,
                         ga_qk_norm=QK_NORM_ALL, ga_rot_half=1, ga_sink=SINK_HEAD, ga_gate=GATE_NONE, ga_scale=float(mix["scale"]),
                         mask_kind=MASK_CAUSAL if size is None else MASK_WINDOW, mask_size=0 if size is None else int(size),
                         **_rotation(mix.get("rot"), f"layer {i}"))
            else:
                raise NotImplementedError(f"layer {i}: mixer type {kind!r}")
            if mlp:
                if mlp.get("kind", "dense") != "dense":
                    raise NotImplementedError(f"layer {i}: feed-forward kind {mlp.get('kind')!r}")
                d.update(ff_kind=FF_GELU, ff=int(mlp["ff"]))
            out.append(d)
        return out


class RamosunForCausalLM(LayerListForCausalLM):
    """Holds the checkpoint tensors (CPU) and builds the device engine on first use.

    dtype: torch.bfloat16 = bf16 matrix products with fp32 accumulation on bf16 weights (norms, convolutions, rotations, scores and
    softmax, gates, memories, the caches and the residual stream in fp32); torch.float32 = everything in true fp32."""
    config_class = RamosunConfig

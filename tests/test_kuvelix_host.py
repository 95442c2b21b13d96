"""CPU checks around Kuvelix: the registry and configuration reader, and properties of the plain oracle that the GPU tests rely on
(causality, rotation and its scaling, both gated units, the router's rules and the identity experts by hand, the looped block)."""
import json
import math

import numpy as np
import pytest

from oracle import kuvelix_oracle as O

AT = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "rot": {"base": 500.0, "dims": 6, "scaling": {"factor": 5.0}}, "scale": 0.4}}
FF = {"kind": "dense", "ff": 20}
MOE = {"kind": "moe", "expert": {"ff": 12, "limit": 1.5}, "router": {"experts": 5, "identity": 3, "groups": {"count": 4, "keep": 2}, "top": 3}}
CFG = {"architecture": "Kuvelix", "width": 32, "vocab": 50, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
       "layers": [dict(AT, mlp=FF), dict(AT, mlp=MOE), dict(AT, mlp=None)]}


def test_registry_and_configuration_reader(tmp_path):
    from llava._b2 import (BLOCK_PARALLEL_RMS, FF_GELU_GLU, FF_MOE, GATE_CHANNEL, MASK_CAUSAL, MIXER_GQA_ATTN, MOE_ACT_CLAMP_GLU, MOE_GROUP_MAX,
                           MOE_SCORE_SOFTMAX, QK_NORM_HEAD, ROT_LINEAR)
    from llava.model import MODEL_REGISTRY, KuvelixConfig, model_class_for

    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert "Kuvelix" in MODEL_REGISTRY and model_class_for(str(tmp_path)).__name__ == "KuvelixForCausalLM"
    c = KuvelixConfig.from_pretrained(str(tmp_path))
    md = c.model_desc()
    assert md["block"] == BLOCK_PARALLEL_RMS and md["embed_norm"] == 1 and md["tied_head"] == 1
    assert (md["loop_start"], md["loop_stop"], md["loop_times"], md["loop_plain"]) == (1, 3, 2, 1)
    a, m, n = c.layer_descs({})
    for x in (a, m, n):
        assert (x["type"], x["ga_heads"], x["ga_kv_heads"], x["ga_dim"], x["ga_vdim"], x["ga_scale"], x["mask_kind"]) == (MIXER_GQA_ATTN, 4, 2, 8, 6, 0.4, MASK_CAUSAL)
        assert (x["ga_qkv_bias"], x["ga_qk_norm"], x["ga_gate"]) == (1, QK_NORM_HEAD, GATE_CHANNEL) and "ga_rot_half" not in x
        assert (x["rot_dims"], x["rot_base"], x["rot_scaling"], x["rot_factor"]) == (6, 500.0, ROT_LINEAR, 5.0)
    assert (a["ff_kind"], a["ff"]) == (FF_GELU_GLU, 20) and n["ff"] == 0
    assert (m["ff_kind"], m["ff"], m["moe_experts"], m["moe_identity"], m["moe_top"], m["moe_groups"], m["moe_keep"]) == (FF_MOE, 12, 5, 3, 3, 4, 2)
    assert (m["moe_act"], m["ff_limit"], m["ff_act_slope"], m["moe_correction"]) == (MOE_ACT_CLAMP_GLU, 1.5, 1.702, 1)
    assert (m["moe_score"], m["moe_group_score"], m["moe_scale"], m.get("moe_raw_weights", 0)) == (MOE_SCORE_SOFTMAX, MOE_GROUP_MAX, 1.0, 0)
    # what a configuration may leave out: loop, rotation, its scaling, kv_heads, groups, identity experts, the limit
    bare = {"architecture": "Kuvelix", "width": 16, "vocab": 9, "norm": {"eps": 1e-6},
            "layers": [{"type": "attention", "mixer": {"heads": 2, "dim": 4, "vdim": 8, "scale": 1.0},
                        "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 4, "top": 2}}},
                       {"type": "attention", "mixer": {"heads": 2, "dim": 4, "vdim": 4, "scale": 1.0, "rot": {"base": 10.0, "dims": 4}}}]}
    b = KuvelixConfig(**bare)
    assert "loop_times" not in b.model_desc()
    bd = b.layer_descs({})
    assert bd[0]["ga_kv_heads"] == 2 and bd[0]["rot_dims"] == 0 and (bd[0]["moe_groups"], bd[0]["moe_keep"], bd[0]["moe_identity"], bd[0]["ff_limit"]) == (1, 1, 0, 0.0)
    assert bd[1]["rot_dims"] == 4 and "rot_factor" not in bd[1] and bd[1]["ff"] == 0
    for key, value in (("type", "mamba"), ("mlp", {"kind": "other"})):
        with pytest.raises(NotImplementedError):
            KuvelixConfig(**dict(bare, layers=[dict(bare["layers"][0], **{key: value})])).layer_descs({})


def test_layer_order_and_shapes():
    assert O.layer_order(CFG) == [0, 1, 2, 1, 2] and O.layer_order(dict(CFG, loop=None)) == [0, 1, 2]
    assert O.layer_order(dict(CFG, loop={"start": 0, "stop": 2, "times": 3})) == [0, 1, 0, 1, 0, 1, 2]
    shapes = O.tensor_shapes(CFG)
    assert shapes["l1.mlp.router"] == (8, 32) and shapes["l1.mlp.correction"] == (8,) and "l1.mlp.e4.up" in shapes and "l1.mlp.e5.up" not in shapes
    assert shapes["l0.mix.g"] == (24, 32) and shapes["l0.mix.k.b"] == (16,) and not any(n.startswith("l2.mlp") for n in shapes)
    logits, layers = O.forward(CFG, O.random_weights(CFG, seed=4), [3, 4, 5, 6], return_layers=True)
    assert layers.shape == (5, 4, 32) and logits.shape == (4, 50)


def test_oracle_is_causal_and_reaches_back_to_the_first_token():
    w = O.random_weights(CFG, seed=1)
    a = list(range(3, 23))
    b = a[:12] + [49 - t for t in a[12:]]
    la, lb = O.forward(CFG, w, a), O.forward(CFG, w, b)
    assert np.allclose(la[:12], lb[:12]) and not np.allclose(la[12:], lb[12:])
    one = dict(CFG, layers=[dict(AT, mlp=None)], loop=None)
    w1 = O.random_weights(one, seed=2)
    assert not np.allclose(O.forward(one, w1, a)[-1], O.forward(one, w1, [40] + a[1:])[-1])


def test_embedding_norm_and_rotation_by_hand():
    w = {"embed": np.array([[0.0, 0.0], [3.0, -4.0]]), "embed.norm": np.array([2.0, 1.0])}
    got = O.embedding({"norm": {"eps": 0.5}}, w, [1, 0])
    assert np.allclose(got, [[6.0 / math.sqrt(13.0), -4.0 / math.sqrt(13.0)], [0.0, 0.0]])
    rot = {"base": 100.0, "dims": 4}
    assert np.allclose(O.rotary_frequencies(rot), [1.0, 0.1]) and np.allclose(O.rotary_frequencies(dict(rot, scaling={"factor": 8.0})), [0.125, 0.0125])
    z = O.rotate_pairs(np.arange(1.0, 7.0), 3, np.array([1.0, 0.1]))
    assert np.allclose(z, [1 * math.cos(3) - 2 * math.sin(3), 2 * math.cos(3) + 1 * math.sin(3), 3 * math.cos(0.3) - 4 * math.sin(0.3),
                           4 * math.cos(0.3) + 3 * math.sin(0.3), 5.0, 6.0])


def test_gated_units_by_hand():
    one = np.eye(1)
    g = O.gelu_tanh(np.array([1.0, -2.0]))
    assert np.allclose(g, [0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715)), -(1 + math.tanh(-math.sqrt(2 / math.pi) * (2 + 0.044715 * 8)))])
    unit = lambda a, b: a / (1 + math.exp(-1.702 * a)) * (b + 1)  # noqa: E731
    for h, gate, up, want in ((1.0, 3.0, 0.5, unit(2.0, 0.5)), (1.0, -9.0, 0.5, unit(-9.0, 0.5)), (1.0, 0.3, 7.0, unit(0.3, 2.0)), (-1.0, 0.3, 7.0, unit(-0.3, -2.0))):
        assert np.allclose(O.expert(np.array([[h]]), gate * one, up * one, one, 2.0), want)
    assert np.allclose(O.expert(np.array([[1.0]]), 3 * one, 7 * one, one, None), unit(3.0, 7.0))


def test_router_rules_by_hand():
    """Eight rows in four groups of two. Scores are given through the logits; every choice is followed by hand."""
    s = np.array([0.30, 0.02, 0.20, 0.05, 0.10, 0.08, 0.15, 0.10])
    r = {"experts": 6, "identity": 2, "groups": {"count": 4, "keep": 2}, "top": 3}
    idx, wgt = O.route(np.ones((1, 1)), np.log(s)[:, None], np.zeros(8), r)
    assert idx[0] == [0, 2, 3] and np.allclose(wgt[0], np.array([0.30, 0.20, 0.05]) / 0.55)
    # a correction moves the choice (row 7 first, group 3 in, group 1 out), never the weights
    c = np.array([0, 0.1, 0, 0, 0, 0, 0, 0.4])
    idx, wgt = O.route(np.ones((1, 1)), np.log(s)[:, None], c, r)
    assert idx[0] == [7, 0, 6] and np.allclose(wgt[0], np.array([0.10, 0.30, 0.15]) / 0.55)
    # all choice scores negative: experts of dropped groups stay out of reach
    idx, _ = O.route(np.ones((1, 1)), np.log(s)[:, None], c - 2.0, r)
    assert idx[0] == [7, 0, 6]
    # identity experts hand their input on
    h = np.array([[2.0, -1.0]])
    p = {"router": np.stack([np.log(s) / 2.0, np.zeros(8)], axis=1), "correction": c}
    for e in range(6):
        p[f"e{e}.gate"], p[f"e{e}.up"], p[f"e{e}.down"] = np.full((1, 2), 0.5), np.zeros((1, 2)), np.array([[1.0], [3.0]]) * (e + 1)
    y = O.moe_ff(h, p, {"expert": {"limit": 9.0}, "router": r})
    unit = 0.5 / (1 + math.exp(-0.851))
    assert np.allclose(y[0], (0.30 / 0.55) * unit * np.array([1.0, 3.0]) + (0.25 / 0.55) * h[0])

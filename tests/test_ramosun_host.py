"""CPU checks around Ramosun: the registry and configuration reader, and properties of the plain oracle that the GPU tests rely on
(causality, the window, the dynamic tanh, banded frequencies by hand, both memories by hand, the sink, the looped block's mix)."""
import json
import math

import numpy as np
import pytest

from oracle import ramosun_oracle as O

BANDS = {"factor": 5.0, "low": 1.0, "high": 4.0, "original": 60}
ML = {"type": "mlstm", "mixer": {"heads": 3, "dim": 4, "vdim": 6, "gate_cap": 9.0}}
DN = {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 8, "conv": 3}}
AT = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 1, "dim": 8, "vdim": 8, "mask": {"size": 5}, "rot": {"base": 500.0, "dims": 6, "scaling": BANDS},
                                     "scale": 0.4}}
FF = {"kind": "dense", "ff": 20}
CFG = {"architecture": "Ramosun", "width": 32, "vocab": 50, "norm": {"eps": 1e-5}, "logit_softcap": 7.0, "loop": {"start": 1, "stop": 3, "times": 2},
       "layers": [dict(AT, mlp=FF), dict(ML, mlp=None), dict(DN, mlp=FF)]}


def test_registry_and_configuration_reader(tmp_path):
    from llava._b2 import (BLOCK_PARALLEL2, FF_GELU, GATE_NONE, MASK_CAUSAL, MASK_WINDOW, MIXER_DELTA, MIXER_GQA_ATTN, MIXER_MLSTM, NORM_DYT, QK_NORM_ALL,
                           ROT_BANDS, SINK_HEAD)
    from llava.model import MODEL_REGISTRY, RamosunConfig, model_class_for

    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert "Ramosun" in MODEL_REGISTRY and model_class_for(str(tmp_path)).__name__ == "RamosunForCausalLM"
    c = RamosunConfig.from_pretrained(str(tmp_path))
    md = c.model_desc()
    assert md["block"] == BLOCK_PARALLEL2 and md["norm_kind"] == NORM_DYT and md["tied_head"] == 1 and md["logit_softcap"] == 7.0
    assert (md["loop_start"], md["loop_stop"], md["loop_times"], md["loop_mix"]) == (1, 3, 2, 1)
    a, m, d = c.layer_descs({})
    assert [x["type"] for x in (a, m, d)] == [MIXER_GQA_ATTN, MIXER_MLSTM, MIXER_DELTA]
    assert (m["ml_heads"], m["ml_dim"], m["ml_vdim"], m["ml_cap"], m["ff"]) == (3, 4, 6, 9.0, 0)
    assert (d["dn_heads"], d["dn_kv_heads"], d["dn_dim"], d["dn_vdim"], d["dn_conv"], d["ff_kind"], d["ff"]) == (4, 2, 6, 8, 3, FF_GELU, 20)
    assert (a["ga_heads"], a["ga_kv_heads"], a["ga_dim"], a["ga_vdim"], a["mask_kind"], a["mask_size"]) == (4, 1, 8, 8, MASK_WINDOW, 5)
    assert a["ga_key_values"] == 1 and a["ga_qk_norm"] == QK_NORM_ALL and a["ga_sink"] == SINK_HEAD and a["ga_rot_half"] == 1 and a["ga_gate"] == GATE_NONE
    assert (a["rot_dims"], a["rot_scaling"], a["rot_factor"], a["rot_original"], a["rot_fast"], a["rot_slow"]) == (6, ROT_BANDS, 5.0, 60.0, 4.0, 1.0)
    # what a configuration may leave out: loop, soft-cap, mask, rotation, kv_heads, the taps (read from the checkpoint)
    bare = {"architecture": "Ramosun", "width": 16, "vocab": 9, "norm": {"eps": 1e-6},
            "layers": [{"type": "attention", "mixer": {"heads": 2, "dim": 4, "scale": 1.0}, "mlp": None},
                       {"type": "delta", "mixer": {"heads": 2, "dim": 4, "vdim": 4}}]}
    b = RamosunConfig(**bare)
    assert "loop_times" not in b.model_desc() and b.model_desc()["logit_softcap"] == 0.0
    bd = b.layer_descs({"l1.mix.q.conv": (8, 5)})
    assert bd[0]["ga_kv_heads"] == 2 and bd[0]["mask_kind"] == MASK_CAUSAL and bd[0]["rot_dims"] == 0 and bd[1]["dn_conv"] == 5 and bd[1]["dn_kv_heads"] == 2
    bare["layers"][0]["mixer"]["vdim"] = 6
    with pytest.raises(ValueError):
        RamosunConfig(**bare).layer_descs({"l1.mix.q.conv": (8, 5)})


def test_layer_order_and_the_mix_of_a_looped_block():
    assert O.layer_order(CFG) == [(0, False), (1, True), (2, False), (1, True), (2, False)]
    assert O.layer_order(dict(CFG, loop={"start": 0, "stop": 1, "times": 1})) == [(0, True), (1, False), (2, False)]
    assert O.layer_order(dict(CFG, loop=None)) == [(0, False), (1, False), (2, False)]
    w = O.random_weights(CFG, seed=4)
    logits, layers = O.forward(CFG, w, [3, 4, 5, 6], return_layers=True)
    assert layers.shape == (5, 4, 32) and logits.shape == (4, 50) and np.abs(logits).max() < 7.0
    x, x0 = np.ones((1, 32)), np.full((1, 32), 2.0)
    m = np.asarray(w["loop.in"], np.float64)
    assert np.allclose(O.open_pass(x, x0, w), (m[:, :32].sum(1) + 2.0 * m[:, 32:].sum(1))[None])


def test_oracle_is_causal_and_keeps_its_window():
    w = O.random_weights(CFG, seed=1)
    a = list(range(3, 23))
    b = a[:12] + [49 - t for t in a[12:]]
    la, lb = O.forward(CFG, w, a), O.forward(CFG, w, b)
    assert np.allclose(la[:12], lb[:12]) and not np.allclose(la[12:], lb[12:])
    assert [j for j in range(12) if O.sees_window(10, j, 4)] == [7, 8, 9, 10] and [j for j in range(4) if O.sees_window(3, j, None)] == [0, 1, 2, 3]
    one = dict(CFG, layers=[dict(AT, mlp=None)], loop=None)
    w1 = O.random_weights(one, seed=2)
    x = O.forward(one, w1, a)
    y = O.forward(one, w1, a[:3] + [a[3] + 1] + a[4:])
    assert not np.allclose(x[7], y[7]) and np.allclose(x[8:], y[8:])          # a window of five: position 3 reaches position 7 and no further


def test_dynamic_tanh_and_gelu():
    w = {"n": np.array([2.0, 1.0]), "n.b": np.array([0.5, -1.0]), "n.alpha": np.array(0.7)}
    assert np.allclose(O.dyt(np.array([[3.0, -2.0]]), w, "n"), [[2.0 * math.tanh(2.1) + 0.5, math.tanh(-1.4) - 1.0]])
    assert np.allclose(O.gelu(np.array([1.0, -2.0])), [0.5 * (1 + math.erf(2 ** -0.5)), -1.0 * (1 + math.erf(-2.0 ** 0.5))])


def test_banded_frequencies_by_hand():
    rot = {"base": 100.0, "dims": 8}
    plain = O.rotary_frequencies(rot)
    assert np.allclose(plain, [1.0, 100 ** -0.25, 0.1, 100 ** -0.75])
    got = O.rotary_frequencies(dict(rot, scaling={"factor": 5.0, "low": 1.0, "high": 4.0, "original": 60}))
    turns = 60 * plain / (2 * math.pi)                       # 9.5, 3.0, 0.95, 0.30
    assert turns[0] > 4 and 1 < turns[1] < 4 and turns[2] < 1 and turns[3] < 1
    s = (turns[1] - 1) / 3
    assert np.allclose(got, [plain[0], (1 - s) * plain[1] / 5 + s * plain[1], plain[2] / 5, plain[3] / 5])
    x = np.arange(1.0, 7.0)
    z = O.rotate_half(x, 3, np.array([1.0, 0.1]))
    assert np.allclose(z, [1 * math.cos(3) - 3 * math.sin(3), 2 * math.cos(0.3) - 4 * math.sin(0.3), 3 * math.cos(3) + 1 * math.sin(3),
                           4 * math.cos(0.3) + 2 * math.sin(0.3), 5.0, 6.0])


def test_mlstm_memory_by_hand():
    """Two steps of one head against the plain sums: with m the running maximum, S exp(m) and n exp(m) are the unscaled memory, so the
    read-out is sum_s w_s (k_s . q) v_s / (max(|sum_s w_s (k_s . q)|, 1) + 1e-6 exp(m)) with w_s = exp(i_s + f_(s+1) + ..)."""
    q, k, v = np.array([[1.0, 2.0], [0.5, -1.0]]), np.array([[0.3, 0.1], [2.0, 1.0]]), np.array([[1.0, 5.0, 2.0], [-1.0, 0.5, 3.0]])
    i, f = np.array([0.7, -2.0]), np.array([-0.4, -0.1])
    got = O.mlstm_memory(q, k, v, i, f)
    m0 = max(-0.4, 0.7)
    d0 = math.exp(0.7) * (k[0] @ q[0])
    assert np.allclose(got[0], d0 * v[0] / (max(abs(d0), 1.0) + 1e-6 * math.exp(m0)))
    m1 = max(m0 - 0.1, -2.0)
    c = [math.exp(0.7 - 0.1) * (k[0] @ q[1]), math.exp(-2.0) * (k[1] @ q[1])]
    assert np.allclose(got[1], (c[0] * v[0] + c[1] * v[1]) / (max(abs(sum(c)), 1.0) + 1e-6 * math.exp(m1)))
    # an input gate far below zero: the maximum starts at 0, so the first token is NOT brought up to weight one
    low = O.mlstm_memory(q[:1], k[:1], v[:1], np.array([-9.0]), np.array([-0.2]))
    assert np.allclose(low[0], math.exp(-9.0) * (k[0] @ q[0]) * v[0] / (1.0 + 1e-6 * math.exp(-0.2)))
    g, h = O.mlstm_gates(np.array([[3.0]]), {"i": np.array([[2.0]]), "i.b": np.array([1.0]), "f": np.array([[1.0]]), "f.b": np.array([0.0])}, {"gate_cap": 4.0})
    assert np.allclose(g, 4 * math.tanh(7 / 4)) and np.allclose(h, -math.log1p(math.exp(-4 * math.tanh(3 / 4))))


def test_delta_memory_by_hand():
    k, q, v = np.array([[1.0, 0.0], [0.6, 0.8]]), np.array([[1.0, 1.0], [2.0, 0.0]]), np.array([[3.0], [5.0]])
    got = O.delta_memory(q, k, v, np.array([1.0, 0.5]), np.array([0.9, 0.5]))
    # full strength: the first key holds its value; then the memory halves, and half of what is missing under the second key is written
    S = np.array([3.0, 0.0])
    assert np.allclose(got[0], S @ q[0])
    S = 0.5 * S
    S = S + k[1] * 0.5 * (5.0 - S @ k[1])
    assert np.allclose(got[1], S @ q[1])
    assert np.allclose(O.unit(np.array([3.0, 4.0])), np.array([0.6, 0.8]), atol=1e-6)


def test_sink_in_the_denominator():
    s, v = np.array([-3.0, -4.0]), np.array([[1.0, 0.0], [0.0, 1.0]])
    e = np.exp(s)
    assert np.allclose(O.softmax_attend(s, v, 0.5), e / (math.exp(0.5) + e.sum())) and np.allclose(O.softmax_attend(s, v, None), e / e.sum())
    big = np.array([50.0, 49.0])
    assert np.allclose(O.softmax_attend(big, v, 52.0), np.exp(big - 52) / (1 + np.exp(big - 52).sum()))

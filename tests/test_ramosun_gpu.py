"""Ramosun on the engine against the plain oracle (oracle/ramosun_oracle.py): every mechanism alone, prompts in one piece, in
portions down to two tokens and token by token, batched decode steps of unequal requests, slots that are freed and used again,
keys far away, at the edges of key tiles and just inside / outside every window (in prompts and in decode steps), the first tokens of
a sequence, long decoding, looped blocks and their input mix, greedy generation through generate() and the continuous batcher, the
replay program. Small configurations whose sizes differ from one another (and from multiples of the kernels' tiles), random weights,
both number formats; where random weights would hide a fault the weights are shaped so that it shows."""
import copy
import threading

import numpy as np
import pytest
import torch

from oracle import ramosun_oracle as O

pytestmark = pytest.mark.gpu

BANDS = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40}


def mlstm(heads, dim, vdim, cap=15.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attn(heads, kv_heads, dim, size, rot_dims, base=500.0, scaling=None, scale=0.3):
    mix = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if size is not None:
        mix["mask"] = {"size": size}
    if rot_dims:
        mix["rot"] = {"base": base, "dims": rot_dims}
        if scaling:
            mix["rot"]["scaling"] = dict(scaling)
    return {"type": "attention", "mixer": mix}


ML = mlstm(3, 16, 24)
ML_ODD = mlstm(5, 9, 7, cap=3.0)                     # nothing a multiple of 4; a cap that bends most gates
ML_ONE = mlstm(1, 40, 16, cap=30.0)                  # one head; its 16 value columns fill a column block, the normaliser opens the next
ML_WIDE = mlstm(2, 136, 44)                          # keys beyond 128
ML_MID = mlstm(2, 100, 31, cap=8.0)                  # the normaliser is the last column of a full block
DN = delta(6, 2, 16, 20, 4)                          # three value heads per q / k head
DN_ODD = delta(3, 3, 7, 9, 2)                        # odd sizes
DN_ONE = delta(1, 1, 48, 4, 1)                       # a convolution of ONE tap: nothing is carried but the memory
DN_WIDE = delta(2, 1, 132, 40, 7)                    # keys beyond 128
DN_MID = delta(4, 2, 72, 33, 3)
AT = attn(6, 2, 16, 11, 8, scaling=BANDS)            # part of a head rotated, frequencies on all three sides of the bands
AT_ODD = attn(2, 2, 9, 4, 6, base=10000.0)           # odd sizes, a rotated part that ends inside the head
AT_ONE = attn(1, 1, 8, 1, 8)                         # one head, a window of the query alone
AT_PLAIN = attn(4, 1, 12, 64, 12, base=1.0e6)        # one key/value head, all of a head rotated
AT_FREE = attn(3, 3, 20, None, 0)                    # no mask and no rotation
AT_WIDE = attn(4, 2, 136, 50, 40, scaling=BANDS, scale=0.1)     # heads wider than 128
FF = {"kind": "dense", "ff": 40}
FF_ODD = {"kind": "dense", "ff": 27}
FF_WIDE = {"kind": "dense", "ff": 136}


def layer(mixer, mlp):
    out = copy.deepcopy(mixer)
    out["mlp"] = copy.deepcopy(mlp)
    return out


def config(layers, width=72, vocab=150, eps=1e-5, cap=20.0, loop=None):
    cfg = {"architecture": "Ramosun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": copy.deepcopy(layers)}
    if cap is not None:
        cfg["logit_softcap"] = cap
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CFG_MAIN = config([layer(AT, FF), layer(ML, FF_WIDE), layer(DN, None), layer(AT_PLAIN, FF)], width=64, vocab=152, loop=(1, 3, 2))
CFG_ODD = config([layer(DN_ODD, FF_ODD), layer(ML_ODD, None), layer(AT_ODD, FF_ODD)], width=50, vocab=77, eps=1e-3, cap=None)
CFG_ONE = config([layer(AT_ONE, None), layer(DN_ONE, FF_WIDE), layer(ML_ONE, FF)], width=48, cap=4.0, loop=(0, 3, 3))
CFG_WIDE = config([layer(ML_WIDE, FF), layer(DN_WIDE, FF), layer(AT_WIDE, None)], width=56, loop=(2, 3, 1))
CFG_MID = config([layer(DN_MID, FF_WIDE), layer(AT_FREE, FF), layer(ML_MID, FF_ODD)], width=80, loop=(1, 2, 2))
ALL_CFGS = [CFG_MAIN, CFG_ODD, CFG_ONE, CFG_WIDE, CFG_MID]
ALL_IDS = ["main", "odd", "one", "wide", "mid"]


def build(cfg, dtype=torch.float32, seed=0, weights=None, **limits):
    from llava.model import RamosunConfig, RamosunForCausalLM

    w = weights if weights is not None else O.random_weights(cfg, seed=seed)
    limits = {"max_batch": 4, "max_seq": 256, **limits}
    model = RamosunForCausalLM(RamosunConfig(**cfg), {k: torch.from_numpy(np.asarray(v, np.float32)).bfloat16() for k, v in w.items()}, dtype=dtype, **limits)
    return model, w


def tokens_for(cfg, n, seed=1):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def row_errors(a, b):
    a = torch.as_tensor(np.asarray(a.detach().cpu() if torch.is_tensor(a) else a), dtype=torch.float64)
    b = torch.as_tensor(np.asarray(b.detach().cpu() if torch.is_tensor(b) else b), dtype=torch.float64)
    return ((a - b) ** 2).mean(-1).sqrt() / (b.std(-1) + 1e-12)


def err(a, b):
    """rms difference over std of the reference, per row, worst row"""
    return float(row_errors(a, b).max())


def close(a, b, dtype, tight=False):
    """fp32: every row within rounding. bf16: nine rows in ten within the format's rounding."""
    e = row_errors(a, b).flatten()
    if dtype == torch.float32:
        return float(e.max()) < (2e-5 if tight else 2e-4)
    return float(torch.quantile(e, 0.9)) < (2e-2 if tight else 6e-2)


def run_schedule(eng, kv, slot, toks, cuts, decode_single=True):
    """Feed toks in portions of the sizes `cuts` (the rest one by one); a single token of a running request takes the decode
    step when decode_single, else the portion call. Returns logits of every position."""
    out, at, first = [], 0, True
    sizes = list(cuts) + [1] * (len(toks) - sum(cuts))
    for n in sizes:
        part = toks[at:at + n]
        if n == 1 and not first and decode_single:
            out.append(eng.decode_step(kv, torch.tensor(part, dtype=torch.int32), slot0=slot))
        else:
            out.append(eng.append_tokens(kv, slot, part, list(range(n)), restart=first))
        at, first = at + n, False
    return torch.cat(out)


# ----------------------------------------------------------------------------------------------------------- mechanisms alone
MIXERS = {"mlstm": ML, "mlstm_odd": ML_ODD, "mlstm_one": ML_ONE, "mlstm_wide": ML_WIDE, "mlstm_mid": ML_MID, "delta": DN, "delta_odd": DN_ODD,
          "delta_one": DN_ONE, "delta_wide": DN_WIDE, "delta_mid": DN_MID, "attn": AT, "attn_odd": AT_ODD, "attn_one": AT_ONE, "attn_plain": AT_PLAIN,
          "attn_free": AT_FREE, "attn_wide": AT_WIDE}
MLPS = {"dense": FF, "dense_odd": FF_ODD, "dense_wide": FF_WIDE}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(MIXERS) + list(MLPS))
def test_each_mechanism_alone(name, dtype):
    """One layer: the residual stream after it equals x + mixer(N1(x)) + ff(N2(x)), built here from the oracle's function for that
    mechanism. A feed-forward is tested beside the smallest mixer."""
    lay = layer(MIXERS.get(name, AT_ONE), MLPS.get(name))
    cfg = config([lay], width=50 if name.endswith("odd") else 72)
    w = O.random_weights(cfg, seed=2)
    model, _ = build(cfg, dtype, weights=w)
    toks = tokens_for(cfg, 75)
    _, hidden = model.forward(torch.tensor([toks]), output_hidden_states=True)
    eps = cfg["norm"]["eps"]
    x = np.asarray(w["embed"], np.float64)[toks]
    y = O.MIXERS[lay["type"]](O.dyt(x, w, "l0.norm1"), O.layer_params(w, 0, "mix"), lay["mixer"], eps)
    if lay["mlp"]:
        y = y + O.feed_forward(O.dyt(x, w, "l0.norm2"), O.layer_params(w, 0, "mlp"))
    assert close(hidden[0, 0], x + y, dtype)


def test_slopes_and_biases_of_every_norm_show():
    """An oracle that takes one norm's slope, weight or bias for another's is far away; the engine agrees with the right one in a
    prompt (normed in a pass of its own) and in decode steps (normed on the way into the products)."""
    cfg = config([layer(AT_PLAIN, FF)], width=64)
    w = O.random_weights(cfg, seed=5)
    for name, al in (("l0.norm1", 0.3), ("l0.norm2", 1.4), ("final.norm", 0.7)):
        w[name + ".alpha"] = O.bf16_round(np.float32(al).reshape(()))
        w[name + ".b"] = O.bf16_round(w[name + ".b"] * 6.0)
    toks = tokens_for(cfg, 60, seed=3)
    ref = O.forward(cfg, w, toks)
    for part in (".alpha", "", ".b"):
        swapped = dict(w)
        swapped["l0.norm1" + part], swapped["l0.norm2" + part] = w["l0.norm2" + part], w["l0.norm1" + part]
        assert float(row_errors(O.forward(cfg, swapped, toks), ref).median()) > 0.03, part or "weight"
    for dtype in (torch.float32, torch.bfloat16):
        model, _ = build(cfg, dtype, weights=w)
        eng = model._ensure_engine()
        kv = eng.new_kv(1, 256)
        assert close(run_schedule(eng, kv, 0, toks, [60]), ref, dtype)
        assert close(run_schedule(eng, kv, 0, toks, [20]), ref, dtype)


# ----------------------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cfg", ALL_CFGS, ids=ALL_IDS)
def test_whole_prompt_against_the_oracle(cfg, dtype):
    model, w = build(cfg, dtype)
    toks = tokens_for(cfg, 150, seed=2)
    logits, hidden = model.forward(torch.tensor([toks]), output_hidden_states=True)
    ref, layers = O.forward(cfg, w, toks, return_layers=True)
    runs = len(O.layer_order(cfg))
    assert hidden.shape == (1, runs, len(toks), cfg["width"])          # a looped layer counts every time
    for i in range(runs):
        assert close(hidden[0, i], layers[i], dtype), f"residual stream after layer run {i}"
    assert close(logits[0], ref, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cfg", ALL_CFGS, ids=ALL_IDS)
def test_portions_and_token_by_token_equal_the_whole_prompt(cfg, dtype):
    model, w = build(cfg, dtype)
    eng = model._ensure_engine()
    kv = eng.new_kv(2, 256)
    toks = tokens_for(cfg, 131, seed=3)
    whole = run_schedule(eng, kv, 0, toks, [len(toks)])
    assert close(whole, O.forward(cfg, w, toks), dtype)
    for cuts in ([1], [2] * 40, [9] * 6, [7, 2, 1, 13, 3, 2, 64, 2], [70, 2, 2, 3], [64, 64], [16, 15, 17, 32, 2]):
        assert close(run_schedule(eng, kv, 1, toks, cuts), whole, dtype, tight=True), f"portions {cuts[:4]}.. then decode steps"
        assert close(run_schedule(eng, kv, 1, toks, cuts, decode_single=False), whole, dtype, tight=True), f"portions {cuts[:4]}.. then portions of one"


def test_the_first_tokens_of_a_sequence():
    """Prompts of one, two and three tokens (shorter than the convolution), alone and continued one by one."""
    cfg = CFG_MAIN
    model, w = build(cfg, torch.float32)
    eng = model._ensure_engine()
    kv = eng.new_kv(2, 256)
    toks = tokens_for(cfg, 12, seed=8)
    ref = O.forward(cfg, w, toks)
    for n in (1, 2, 3):
        assert err(run_schedule(eng, kv, 0, toks[:n], [n]), ref[:n]) < 2e-4
        assert err(run_schedule(eng, kv, 0, toks, [n]), ref) < 2e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_decoding_moves_windows_and_memories_over_decoded_tokens(dtype):
    cfg = CFG_MAIN
    model, w = build(cfg, dtype)
    eng = model._ensure_engine()
    kv = eng.new_kv(2, 256)
    toks = tokens_for(cfg, 170, seed=5)
    got = run_schedule(eng, kv, 0, toks, [8])          # 162 decode steps: every window passes over decoded tokens many times
    ref = O.forward(cfg, w, toks)
    assert close(got[-40:], ref[-40:], dtype)
    assert close(got, ref, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cfg", [CFG_MAIN, CFG_MID], ids=["main", "mid"])
def test_batched_decode_of_unequal_requests_equals_each_alone(cfg, dtype):
    model, w = build(cfg, dtype, max_batch=12)
    eng = model._ensure_engine()
    kv = eng.new_kv(12, 256)
    steps = 12
    for lengths in ((37, 14), (37, 14, 21, 50, 13), (13, 40, 22, 31, 14, 15, 16, 17, 45, 19)):     # 2, 5 and 10 rows: each takes other Linear kernels
        reqs = [tokens_for(cfg, n, seed=10 + n) for n in lengths]
        alone = [run_schedule(eng, kv, 11, r, [len(r) - steps]) for r in reqs]      # slot 11, one request after the other
        for b, r in enumerate(reqs):
            eng.append_tokens(kv, b, r[:len(r) - steps], [], restart=True)
        got = [[] for _ in reqs]
        for s in range(steps):                                                    # one decode step over the slots
            col = torch.tensor([r[len(r) - steps + s] for r in reqs], dtype=torch.int32)
            lg = eng.decode_step(kv, col)
            for b in range(len(reqs)):
                got[b].append(lg[b])
        for b, r in enumerate(reqs):
            assert close(torch.stack(got[b]), alone[b][-steps:], dtype, tight=True), f"request {b} of {len(reqs)}"
        assert close(torch.stack(got[1]), O.forward(cfg, w, reqs[1])[-steps:], dtype)


def test_a_slot_that_is_freed_and_used_again_starts_clean():
    cfg = CFG_MAIN
    model, w = build(cfg, torch.float32)
    eng = model._ensure_engine()
    kv = eng.new_kv(2, 256)
    a, b = tokens_for(cfg, 90, seed=21), tokens_for(cfg, 33, seed=22)
    fresh = run_schedule(eng, kv, 1, b, [20])
    run_schedule(eng, kv, 0, a, [50])                      # leaves cache rows, memories, running maxima and convolution tails behind
    kv.free_slot(0)
    assert kv.lengths(2)[0] == 0
    again = run_schedule(eng, kv, 0, b, [20])
    assert err(again, fresh) < 1e-6
    third = run_schedule(eng, kv, 0, b, [2, 2])            # restart on a slot that was not freed, shortest portions
    assert err(third, fresh) < 2e-5
    with pytest.raises(ValueError):
        eng.append_tokens(kv, 0, [0] * 300, [], restart=False)   # beyond the slot's capacity


def test_every_pass_of_a_looped_layer_has_its_own_state():
    """Three passes over all three layers against an oracle that runs nine layers with the same tensors and mixes its input in front
    of every third: equal only if no pass shares a cache, a memory or a convolution tail with another, in a prompt, in portions and in
    decode steps. Premise: leaving one mix out, or mixing in the residual stream instead of the embedding output, is far away."""
    cfg = CFG_ONE
    w = O.random_weights(cfg, seed=0)
    toks = tokens_for(cfg, 60, seed=6)
    x0 = np.asarray(w["embed"], np.float64)[toks]

    def unrolled(mix):
        x = x0
        for p in range(3):
            x = mix(p, x)
            for i in range(3):
                x = O.layer_step(x, cfg, w, i)
        return O.head(x, cfg, w)

    ref = O.forward(cfg, w, toks)
    assert np.allclose(ref, unrolled(lambda p, x: O.open_pass(x, x0, w)))
    assert float(row_errors(unrolled(lambda p, x: O.open_pass(x, x0, w) if p else x), ref).median()) > 0.05
    assert float(row_errors(unrolled(lambda p, x: O.open_pass(x, x, w)), ref).median()) > 0.05
    assert float(row_errors(unrolled(lambda p, x: O.open_pass(x0, x, w)), ref).median()) > 0.05
    model, _ = build(cfg, torch.float32, weights=w)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 256)
    for cuts in ([60], [13, 2, 20], [2]):
        assert err(run_schedule(eng, kv, 0, toks, cuts), ref) < 2e-4


# ----------------------------------------------------------------------------------------------------------- edges
def sharp_model(size, seed=7, sink=None):
    """One attention layer whose score factor is scaled up until the softmax is almost an argmax: for most positions ONE visible key
    carries the output, as often the oldest visible one as any other. A key too many or too few at the edge of the window (or of a key
    tile of 32, a key split, a portion) then moves many rows by far more than the tolerance."""
    cfg = config([layer(attn(4, 2, 16, size, 8, base=50.0, scale=3.0), None)], width=48, vocab=400, cap=None)
    w = O.random_weights(cfg, seed=seed)
    w["l0.mix.sink"] = O.bf16_round(np.full(4, -60.0 if sink is None else sink))
    w["l0.mix.k"] = O.bf16_round(w["l0.mix.k"] * 3.0)       # larger values: the mixer's share of the residual stream grows (the keys are normed)
    return cfg, w


@pytest.mark.parametrize("size", [2, 29, 37, 64, 100, 300])
def test_keys_just_inside_and_outside_the_window_and_far_away(size):
    T = 420
    cfg, w = sharp_model(size)
    toks = tokens_for(cfg, T, seed=9)
    ref = O.forward(cfg, w, toks)
    # the test's premise: a window one position larger or smaller changes rows by much more than the tolerance (small windows: every row has
    # an edge close by), and keys further back than a third of a large window carry many rows
    for other in (size - 1, size + 1) if size < 100 else (size // 3,):
        cfg2 = copy.deepcopy(cfg)
        cfg2["layers"][0]["mixer"]["mask"]["size"] = other
        moved = row_errors(O.forward(cfg2, w, toks), ref)
        assert int((moved > 2e-2).sum()) >= (8 if size < 100 else 40), f"a window of {other} instead of {size} would hardly show"
    model, _ = build(cfg, torch.float32, weights=w, max_batch=2, max_seq=1024, max_rows=512)
    eng = model._ensure_engine()
    kv = eng.new_kv(2, 1024)
    assert err(run_schedule(eng, kv, 0, toks, [T]), ref) < 2e-4, "whole prompt"
    assert err(run_schedule(eng, kv, 1, toks, [31, 2, 33, 64, 1, 5, 2, 2, 130]), ref) < 2e-4, "portions that end at and around tile edges, then decode steps"
    assert err(run_schedule(eng, kv, 1, toks, [max(1, size - 1), 2, 2, 64, 3]), ref) < 2e-4, "portions that end just inside and outside the first window edge"
    assert err(run_schedule(eng, kv, 0, toks, [300]), ref) < 2e-4, "120 decode steps over split keys"
    assert err(run_schedule(eng, kv, 1, toks, [max(2, size - 2)]), ref) < 2e-4, "decode steps from just inside the first window edge on"


def test_the_sinks_of_the_softmax_show():
    """A different sink per head, high enough to take most of the weight of many rows. Premise: an oracle without sinks, with the sinks of
    other heads, or whose sink is scaled like a score is far away; the engine agrees with the right one in a prompt and in decode steps
    over split keys."""
    cfg, w = sharp_model(40)
    cfg["layers"][0]["mixer"]["scale"] = 0.5
    w["l0.mix.sink"] = O.bf16_round(np.array([1.0, 4.0, -2.0, 6.0]))
    toks = tokens_for(cfg, 150, seed=12)
    ref = O.forward(cfg, w, toks)
    for other in (np.full(4, -60.0), w["l0.mix.sink"][::-1], w["l0.mix.sink"] * 0.5):
        assert int((row_errors(O.forward(cfg, dict(w, **{"l0.mix.sink": other}), toks), ref) > 0.05).sum()) >= 60
    model, _ = build(cfg, torch.float32, weights=w)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 256)
    assert err(run_schedule(eng, kv, 0, toks, [150]), ref) < 2e-4
    assert err(run_schedule(eng, kv, 0, toks, [20]), ref) < 2e-4


def test_the_values_are_the_raw_keys_and_the_norm_spans_all_heads():
    """Key heads of very different sizes: an oracle that norms every head on its own, takes the normed keys as values, or norms after the
    rotation is far away."""
    cfg = config([layer(attn(4, 2, 12, 30, 12, base=30.0, scale=0.6), None)], width=40, cap=None)
    w = O.random_weights(cfg, seed=3)
    for n, heads in (("q", 4), ("k", 2)):
        m = w[f"l0.mix.{n}"].reshape(heads, 12, -1) * np.array([3.0, 0.3, 1.0, 0.1][:heads])[:, None, None]
        w[f"l0.mix.{n}"] = O.bf16_round(m.reshape(heads * 12, -1))
    w["l0.mix.q.norm"] = O.bf16_round(np.linspace(0.3, 2.0, 48))
    toks = tokens_for(cfg, 90, seed=4)
    ref = O.forward(cfg, w, toks)
    h = O.dyt(np.asarray(w["embed"], np.float64)[toks], w, "l0.norm1")
    p, mix = O.layer_params(w, 0, "mix"), cfg["layers"][0]["mixer"]
    T, f = len(toks), O.rotary_frequencies(mix["rot"])

    def variant(norm_heads=False, normed_values=False):
        raw_q, raw_k = h @ p["q"].T, h @ p["k"].T
        if norm_heads:
            q = O.rms_unit(raw_q.reshape(T, 4, 12), 1e-5) * p["q.norm"].reshape(4, 12)
            k = O.rms_unit(raw_k.reshape(T, 2, 12), 1e-5) * p["k.norm"].reshape(2, 12)
        else:
            q, k = (O.rms_unit(raw_q, 1e-5) * p["q.norm"]).reshape(T, 4, 12), (O.rms_unit(raw_k, 1e-5) * p["k.norm"]).reshape(T, 2, 12)
        v = k if normed_values else raw_k.reshape(T, 2, 12)
        q, k = (np.stack([O.rotate_half(x[t], t, f) for t in range(T)]) for x in (q, k))
        out = np.stack([[O.softmax_attend(k[max(0, i - 29):i + 1, a // 2] @ q[i, a] * 0.6, v[max(0, i - 29):i + 1, a // 2], float(p["sink"][a])) for a in range(4)]
                        for i in range(T)])
        return out.reshape(T, 48) @ p["o"].T

    right = O.attention(h, p, mix, 1e-5)
    assert np.allclose(variant(), right)
    assert float(row_errors(variant(norm_heads=True), right).median()) > 0.05
    assert float(row_errors(variant(normed_values=True), right).median()) > 0.05
    model, _ = build(cfg, torch.float32, weights=w)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 256)
    assert err(run_schedule(eng, kv, 0, toks, [90]), ref) < 2e-4
    assert err(run_schedule(eng, kv, 0, toks, [33, 2, 40]), ref) < 2e-4


@pytest.mark.parametrize("kind", ["mlstm", "delta"])
def test_memories_keep_far_tokens_and_forget_by_their_gates(kind):
    """Gates set so that some heads keep hundreds of tokens and others a few: an oracle that starts its memory 150 tokens late, or forgets
    a little faster, is far away from the last rows; the engine agrees with the right one in a prompt, in portions whose edges fall inside
    the token tiles, and in decode steps."""
    lay = layer(mlstm(4, 24, 20, cap=12.0) if kind == "mlstm" else delta(4, 2, 24, 20, 3), None)
    cfg = config([lay], width=40, vocab=300, cap=None)
    w = O.random_weights(cfg, seed=8)
    slow = dict(w)
    if kind == "mlstm":
        w["l0.mix.f.b"], w["l0.mix.f"] = O.bf16_round(np.array([9.0, 6.0, 3.0, 0.0])), O.bf16_round(w["l0.mix.f"] * 0.5)
        slow = dict(w, **{"l0.mix.f.b": w["l0.mix.f.b"] - 2.0})
    else:
        w["l0.mix.A_log"], w["l0.mix.dt_bias"] = O.bf16_round(np.array([-6.0, -5.0, -3.0, 0.0])), O.bf16_round(np.full(4, -1.0))
        w["l0.mix.b"] = O.bf16_round(w["l0.mix.b"] - 0.3)
        slow = dict(w, **{"l0.mix.A_log": w["l0.mix.A_log"] + 2.0})
    T = 330
    toks = tokens_for(cfg, T, seed=9)
    ref = O.forward(cfg, w, toks)
    assert float(row_errors(O.forward(cfg, w, toks[150:])[-40:], ref[-40:]).median()) > 0.01
    assert float(row_errors(O.forward(cfg, slow, toks)[-40:], ref[-40:]).median()) > 0.01
    model, _ = build(cfg, torch.float32, weights=w, max_seq=512, max_rows=512)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 512)
    assert err(run_schedule(eng, kv, 0, toks, [T]), ref) < 2e-4
    assert err(run_schedule(eng, kv, 0, toks, [15, 2, 16, 17, 1, 33, 2, 100]), ref) < 2e-4
    assert err(run_schedule(eng, kv, 0, toks, [200]), ref) < 2e-4


def test_gates_far_out_keep_the_memory_in_range():
    """Input gates near their cap of 40 (their exponential overflows fp32 several times over once summed) and forget gates that close:
    the running maximum carries it. The floor exp(-m) of the normaliser shows where |n . q| is small (input gates far below zero)."""
    lay = layer(mlstm(2, 12, 10, cap=40.0), None)
    cfg = config([lay], width=40, vocab=200, cap=None)
    w = O.random_weights(cfg, seed=18)
    w["l0.mix.i.b"], w["l0.mix.i"] = O.bf16_round(np.array([60.0, -25.0])), O.bf16_round(w["l0.mix.i"] * 30.0)
    w["l0.mix.f.b"], w["l0.mix.f"] = O.bf16_round(np.array([4.0, 30.0])), O.bf16_round(w["l0.mix.f"] * 6.0)
    toks = tokens_for(cfg, 140, seed=19)
    ref, layers = O.forward(cfg, w, toks, return_layers=True)
    h = O.dyt(np.asarray(w["embed"], np.float64)[toks], w, "l0.norm1")
    i, _ = O.mlstm_gates(h, O.layer_params(w, 0, "mix"), lay["mixer"])
    assert i[:, 0].max() > 36 and i[:, 1].min() < -30
    model, _ = build(cfg, torch.float32, weights=w)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 256)
    # the gates' arguments run into the tens, so their fp32 rounding is a few 1e-6 relative: wider than elsewhere
    for cuts in ([140], [17, 2, 50], [3]):
        assert err(run_schedule(eng, kv, 0, toks, cuts), ref) < 1e-3


def test_the_delta_rule_overwrites_what_a_key_held():
    """Keys that repeat (a vocabulary of four tokens, no convolution beyond one tap): the write replaces the value stored under the key.
    Premise: an additive memory is far away."""
    cfg = config([layer(delta(2, 1, 8, 12, 1), None)], width=32, vocab=4, cap=None)
    w = O.random_weights(cfg, seed=28)
    w["l0.mix.A_log"] = O.bf16_round(np.array([-8.0, -8.0]))
    toks = tokens_for(cfg, 120, seed=29)
    h = O.dyt(np.asarray(w["embed"], np.float64)[toks], w, "l0.norm1")
    p, mix = O.layer_params(w, 0, "mix"), cfg["layers"][0]["mixer"]
    right = O.delta(h, p, mix, 1e-5)
    q, k, v = (O.silu(O.causal_conv(h @ p[n].T, p[n + ".conv"])) for n in "qkv")
    q, k, v = O.unit(q), O.unit(k), v.reshape(-1, 2, 12)
    beta = O.sigmoid(h @ p["b"].T)
    add = np.stack([np.stack([sum(beta[s, a] * (k[s] @ q[t]) * v[s, a] for s in range(t + 1)) for a in range(2)]) for t in range(60)])
    y = (O.rms_unit(add, 1e-5) * p["norm"] * O.silu(h[:60] @ p["g"].T).reshape(60, 2, 12)).reshape(60, 24) @ p["o"].T
    assert float(row_errors(y[20:], right[20:60]).median()) > 0.1
    ref = O.forward(cfg, w, toks)
    model, _ = build(cfg, torch.float32, weights=w)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 256)
    for cuts in ([120], [30, 2], [2]):
        assert err(run_schedule(eng, kv, 0, toks, cuts), ref) < 2e-4


def test_positions_far_along_keep_their_angles():
    """Rotations at positions in the thousands (angles of thousands of radians at the fastest pair), scaled by bands and plain."""
    cfg = config([layer(attn(2, 1, 8, 6, 8, base=20.0, scaling=BANDS), None), layer(attn(2, 1, 8, 5, 8, base=20.0), None)], width=32, vocab=60)
    model, w = build(cfg, torch.float32, max_seq=4096, max_rows=4096, max_batch=1)
    toks = tokens_for(cfg, 3500, seed=41)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 4096)
    got = run_schedule(eng, kv, 0, toks, [3490])
    ref = O.forward(cfg, w, toks)[-40:]        # windows of a few positions keep the oracle's loops short
    assert err(got[-40:], ref) < 2e-4


def test_the_soft_cap_bends_the_logits():
    cfg = copy.deepcopy(CFG_ODD)
    cfg["logit_softcap"] = 1.5
    model, w = build(cfg, torch.float32)
    toks = tokens_for(cfg, 40, seed=42)
    got, ref = model.forward(torch.tensor([toks]))[0], O.forward(cfg, w, toks)
    assert float(np.abs(ref).max()) <= 1.5 and float(row_errors(O.forward(CFG_ODD, w, toks), ref).median()) > 0.3
    assert err(got, ref) < 2e-4


# ----------------------------------------------------------------------------------------------------------- generation
def greedy_matches_oracle(cfg, w, prompt, new_tokens, tol_margin=1e-3):
    """The generated ids, fed to the oracle, are its own greedy choices wherever its top-2 margin is not a rounding matter."""
    seq = list(prompt) + list(new_tokens)
    ref = torch.from_numpy(O.forward(cfg, w, seq))
    for i, t in enumerate(new_tokens):
        row = ref[len(prompt) - 1 + i]
        top = torch.topk(row, 2)
        if float(top.values[0] - top.values[1]) > tol_margin * float(row.std()):
            assert int(top.indices[0]) == int(t), f"token {i}"


def test_greedy_generation_through_generate():
    cfg = CFG_MAIN
    model, w = build(cfg, torch.float32)
    prompts = torch.tensor([tokens_for(cfg, 12, seed=51), tokens_for(cfg, 12, seed=52)])
    out = model.generate(prompts, max_new_tokens=24)       # past the first window edge
    assert out.shape == (2, 36) and torch.equal(out[:, :12], prompts)
    for b in range(2):
        greedy_matches_oracle(cfg, w, prompts[b].tolist(), out[b, 12:].tolist())
    solo = model.generate(prompts[1:2], max_new_tokens=24)
    assert torch.equal(solo[0], out[1])


def test_continuous_batching_of_unequal_requests():
    """Six generate() threads on three slots: requests join and leave between steps, slots are reused, and every request gets
    the ids it gets alone."""
    cfg = copy.deepcopy(CFG_MAIN)
    model, w = build(cfg, torch.float32)
    prompts = [torch.tensor([tokens_for(cfg, n, seed=60 + n)]) for n in (5, 19, 9, 30, 3, 14)]
    new = [6, 14, 9, 4, 12, 8]
    solo = [model.generate(p, max_new_tokens=n) for p, n in zip(prompts, new)]
    model.invalidate_engine()
    model.config.raw["b2_continuous_batching"] = 3
    results, errors = [None] * len(prompts), []

    def work(i):
        try:
            results[i] = model.generate(prompts[i], max_new_tokens=new[i])
        except BaseException as e:  # noqa: BLE001
            errors.append(e)

    threads = [threading.Thread(target=work, args=(i,)) for i in range(len(prompts))]
    for t in threads:
        t.start()
    for t in threads:
        t.join(timeout=120)
    assert not errors, errors
    stats = model._batcher.stats
    for i in range(len(prompts)):
        assert torch.equal(results[i], solo[i]), f"request {i}"
    assert stats["admitted"] == 6 and stats["max_active"] <= 3 and stats["rows_stepped"] > stats["steps"]
    greedy_matches_oracle(cfg, w, prompts[1][0].tolist(), results[1][0, 19:].tolist())
    model.invalidate_engine()


def test_sampled_generation_repeats_with_the_seed_and_rejects_bad_input():
    cfg = CFG_ODD
    model, _ = build(cfg, torch.bfloat16)
    p = torch.tensor([tokens_for(cfg, 8, seed=71)])
    torch.manual_seed(5)
    a = model.generate(p, do_sample=True, temperature=0.9, top_k=20, top_p=0.95, max_new_tokens=12)
    torch.manual_seed(5)
    b = model.generate(p, do_sample=True, temperature=0.9, top_k=20, top_p=0.95, max_new_tokens=12)
    assert torch.equal(a, b) and int(a.max()) < cfg["vocab"]
    with pytest.raises(ValueError):
        model.generate(torch.tensor([[cfg["vocab"] + 3, 1, 2]]), max_new_tokens=2)
    with pytest.raises(ValueError):
        model.generate(p, max_new_tokens=4000)


def test_a_checkpoint_without_its_tensors_is_refused():
    for cfg, names in ((CFG_ODD, ("l0.mix.A_log", "l1.mix.f.b", "l2.mix.sink", "l2.norm2.alpha", "final.norm.b")), (CFG_ONE, ("loop.in", "l1.mix.v.conv"))):
        w = O.random_weights(cfg, seed=0)
        for missing in names:
            model, _ = build(cfg, torch.float32, weights={k: v for k, v in w.items() if k != missing})
            with pytest.raises(Exception, match=missing.replace(".", r"\.")):
                model._ensure_engine()


# ----------------------------------------------------------------------------------------------------------- the replay program
def write_checkpoint(path, cfg, weights):
    import json
    import os
    import struct

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for k, v in weights.items():
        raw = torch.from_numpy(np.asarray(v, np.float32)).bfloat16().contiguous().view(torch.int16).numpy().tobytes()
        header[k] = {"dtype": "BF16", "shape": list(np.asarray(v).shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program_on_a_written_checkpoint(dtype, tmp_path, repo_root):
    """bin/trace_run on a checkpoint directory: two requests one after the other on slots that are given back, portions down to two
    tokens, single tokens through the decode step, steps that want nothing; every written row against the oracle."""
    import json
    import subprocess
    import sys

    cfg = CFG_MAIN
    w = O.random_weights(cfg, seed=13)
    write_checkpoint(str(tmp_path / "model"), cfg, w)
    a, b = tokens_for(cfg, 60, seed=31), tokens_for(cfg, 23, seed=32)
    steps, want_rows, at = [], [], 0
    for n in (17, 2, 30, 2):                                                   # request a in portions, the last but one asks for nothing
        want = [] if n == 30 else list(range(0, n, 3))
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": a[at:at + n], "want": want}], "end": []})
        want_rows.append(("a", [at + i for i in want]))
        at += n
    for t in range(at, len(a)):                                                # then token by token
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": [a[t]], "want": [0]}], "end": ["a"] if t == len(a) - 1 else []})
        want_rows.append(("a", [t]))
    steps.append({"step": len(steps), "entries": [{"id": "b", "tokens": b, "want": [0, len(b) - 1]}], "end": ["b"]})
    want_rows.append(("b", [0, len(b) - 1]))
    out = tmp_path / "out"
    run = subprocess.run([sys.executable, f"{repo_root}/bin/trace_run", "--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(out),
                          "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [ln for ln in run.stdout.splitlines() if ln.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    ref = {"a": O.forward(cfg, w, a), "b": O.forward(cfg, w, b)}
    got, exp = [], []
    for i, (rid, rows) in enumerate(want_rows):
        path = out / f"{i}.f32"
        if not rows:
            assert not path.exists()
            continue
        got.append(np.fromfile(path, dtype="<f4").reshape(len(rows), cfg["vocab"]))
        exp.append(ref[rid][rows])
    assert close(torch.from_numpy(np.concatenate(got)), np.concatenate(exp), torch.float32 if dtype == "float32" else torch.bfloat16)

"""Kuvelix on the engine against the plain oracle (oracle/kuvelix_oracle.py): every mechanism alone, prompts in one piece, in
portions down to two tokens and token by token, batched decode steps of unequal requests, slots that are freed and used again,
keys far away and at the edges of key tiles and key splits (in prompts and in decode steps), the first tokens of a sequence, long
decoding, looped blocks, the router's choice (corrections of either sign, groups, identity experts) and the experts' bounds, greedy
generation through generate() and the continuous batcher, the replay program. Small configurations whose sizes differ from one another
(and from multiples of the kernels' tiles), random weights, both number formats; where random weights would hide a fault the weights
are shaped so that it shows."""
import copy
import math
import threading

import numpy as np
import pytest
import torch

from oracle import kuvelix_oracle as O

pytestmark = pytest.mark.gpu


def attn(heads, kv_heads, dim, vdim, rot_dims, base=500.0, factor=None, scale=0.3):
    mix = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot_dims:
        mix["rot"] = {"base": base, "dims": rot_dims}
        if factor:
            mix["rot"]["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": mix}


def moe(experts, top, ff, identity=0, groups=None, limit=None):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = dict(zip(("count", "keep"), groups))
    return {"kind": "moe", "expert": {"ff": ff} if limit is None else {"ff": ff, "limit": limit}, "router": r}


AT = attn(6, 2, 16, 24, 8, factor=3.0)               # part of a head rotated, slowed down; values wider than keys
AT_ODD = attn(2, 2, 9, 7, 5, base=10000.0)           # odd sizes, a rotated part of odd size (its last entry passes)
AT_ONE = attn(1, 1, 8, 4, 8, factor=0.5)             # one head, rotated faster instead of slower
AT_PLAIN = attn(4, 1, 12, 20, 12, base=1.0e6)        # one key/value head, all of a head rotated, plain frequencies
AT_FREE = attn(3, 3, 20, 12, 0)                      # no rotation, a key/value head per query head
AT_WIDE = attn(4, 2, 136, 264, 40, factor=8.0, scale=0.1)      # heads wider than 128 and values wider than 256
AT_TILE = attn(8, 2, 64, 32, 64, factor=2.0, scale=0.15)       # sizes the tensor-core products take
AT_MANY = attn(40, 1, 8, 8, 4)                       # more query heads on a key/value head than a tile of rows holds
FF = {"kind": "dense", "ff": 40}
FF_ODD = {"kind": "dense", "ff": 27}
FF_WIDE = {"kind": "dense", "ff": 136}
MOE = moe(9, 3, 24, identity=3, groups=(4, 2), limit=1.0)      # groups that span experts and identity experts
MOE_ODD = moe(7, 4, 13, identity=3, groups=(5, 3), limit=0.5)
MOE_BARE = moe(5, 1, 40)                             # one choice, one group, no identity experts, no bounds
MOE_ALL = moe(4, 6, 16, identity=2, groups=(3, 3), limit=3.0)  # everything is chosen
MOE_IDLE = moe(2, 2, 32, identity=14, groups=(2, 1), limit=1.5)    # mostly identity experts; a group of identity experts alone
MOE_WIDE = moe(33, 5, 48, identity=7, groups=(10, 4), limit=0.7)   # more router rows than a warp


def layer(mixer, mlp):
    out = copy.deepcopy(mixer)
    out["mlp"] = copy.deepcopy(mlp)
    return out


def config(layers, width=72, vocab=150, eps=1e-5, loop=None):
    cfg = {"architecture": "Kuvelix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": copy.deepcopy(layers)}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CFG_MAIN = config([layer(AT, FF), layer(AT_PLAIN, MOE), layer(AT, None), layer(AT_FREE, MOE_BARE)], width=64, vocab=152, loop=(1, 3, 2))
CFG_ODD = config([layer(AT_ODD, MOE_ODD), layer(AT_ODD, FF_ODD), layer(AT_ODD, None)], width=50, vocab=77, eps=1e-3)
CFG_ONE = config([layer(AT_ONE, MOE_ALL), layer(AT_PLAIN, FF_WIDE)], width=48, loop=(0, 2, 3))
CFG_WIDE = config([layer(AT_WIDE, MOE_IDLE), layer(AT_MANY, FF)], width=56, loop=(1, 2, 1))
CFG_TILE = config([layer(AT_TILE, FF_WIDE), layer(AT_TILE, MOE_WIDE)], width=96, vocab=200, loop=(1, 2, 2))
ALL_CFGS = [CFG_MAIN, CFG_ODD, CFG_ONE, CFG_WIDE, CFG_TILE]
ALL_IDS = ["main", "odd", "one", "wide", "tile"]


def build(cfg, dtype=torch.float32, seed=0, weights=None, **limits):
    from llava.model import KuvelixConfig, KuvelixForCausalLM

    w = weights if weights is not None else O.random_weights(cfg, seed=seed)
    limits = {"max_batch": 4, "max_seq": 256, **limits}
    model = KuvelixForCausalLM(KuvelixConfig(**cfg), {k: torch.from_numpy(np.asarray(v, np.float32)).bfloat16() for k, v in w.items()}, dtype=dtype, **limits)
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
MIXERS = {"attn": AT, "attn_odd": AT_ODD, "attn_one": AT_ONE, "attn_plain": AT_PLAIN, "attn_free": AT_FREE, "attn_wide": AT_WIDE, "attn_tile": AT_TILE,
          "attn_many": AT_MANY}
MLPS = {"dense": FF, "dense_odd": FF_ODD, "dense_wide": FF_WIDE, "moe": MOE, "moe_odd": MOE_ODD, "moe_bare": MOE_BARE, "moe_all": MOE_ALL,
        "moe_idle": MOE_IDLE, "moe_wide": MOE_WIDE}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(MIXERS) + list(MLPS))
def test_each_mechanism_alone(name, dtype):
    """One layer: the residual stream after it equals x + mixer(u) + ff(u), built here from the oracle's function for that mechanism. A
    feed-forward is tested beside the smallest mixer. In a prompt, in one-row steps, and in steps of three and nine rows."""
    lay = layer(MIXERS.get(name, AT_ONE), MLPS.get(name))
    cfg = config([lay], width=50 if name.endswith("odd") else 72)
    w = O.random_weights(cfg, seed=2)
    model, _ = build(cfg, dtype, weights=w)
    toks = tokens_for(cfg, 75)
    logits, hidden = model.forward(torch.tensor([toks]), output_hidden_states=True)
    eps = cfg["norm"]["eps"]
    x = O.embedding(cfg, w, toks)
    u = O.rms_norm(x, w["l0.norm1"], eps)
    y = O.attention(u, O.layer_params(w, 0, "mix"), lay["mixer"], eps)
    if lay["mlp"]:
        y = y + O.feed_forward(u, O.layer_params(w, 0, "mlp"), lay["mlp"])
    assert close(hidden[0, 0], x + y, dtype)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 256)
    for cuts in ([64], [3] * 25, [9] * 8):
        assert close(run_schedule(eng, kv, 0, toks, cuts), logits[0], dtype, tight=True), cuts[:2]


def logits_agree(cfg, w, toks, ref, schedules, tol=2e-4):
    model, _ = build(cfg, torch.float32, weights=w, max_seq=512, max_rows=512)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 512)
    for cuts in schedules:
        assert err(run_schedule(eng, kv, 0, toks, cuts), ref) < tol, cuts[:4]
    model, _ = build(cfg, torch.bfloat16, weights=w, max_seq=512, max_rows=512)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 512)
    for cuts in schedules:
        assert close(run_schedule(eng, kv, 0, toks, cuts), ref, torch.bfloat16), cuts[:4]


def test_the_embedding_is_normed_and_both_sublayers_read_one_norm():
    """Table rows of very different lengths; premise: an oracle without the embedding's norm, or whose feed-forward reads the stream after
    the mixer, is far away."""
    cfg = config([layer(AT_PLAIN, FF)], width=64)
    w = O.random_weights(cfg, seed=5)
    w["embed"] = O.bf16_round(w["embed"] * np.linspace(0.2, 5.0, cfg["vocab"])[:, None])
    toks = tokens_for(cfg, 70, seed=3)
    ref = O.forward(cfg, w, toks)
    eps = cfg["norm"]["eps"]

    def variant(normed, parallel):
        x = O.embedding(cfg, w, toks) if normed else np.asarray(w["embed"], np.float64)[toks]
        u = O.rms_norm(x, w["l0.norm1"], eps)
        y = x + O.attention(u, O.layer_params(w, 0, "mix"), cfg["layers"][0]["mixer"], eps)
        y = y + O.dense_ff(u if parallel else O.rms_norm(y, w["l0.norm1"], eps), O.layer_params(w, 0, "mlp"))
        return O.rms_norm(y, w["final.norm"], eps) @ np.asarray(w["embed"], np.float64).T

    assert np.allclose(variant(True, True), ref)
    assert float(row_errors(variant(False, True), ref).median()) > 0.05
    assert float(row_errors(variant(True, False), ref).median()) > 0.05
    logits_agree(cfg, w, toks, ref, ([70], [20, 2, 9], [1]))


def test_biases_and_head_norms_show():
    """Large biases, different on q, k and v; weights of the two head norms far apart. Premise: an oracle without one bias, with the k
    bias behind the norm, or with the two norms exchanged is far away."""
    cfg = config([layer(attn(4, 2, 16, 16, 8, base=30.0, scale=0.5), None)], width=64)
    w = O.random_weights(cfg, seed=6)
    for n, f in (("q", 3.0), ("k", 2.0), ("v", 2.5)):
        w[f"l0.mix.{n}.b"] = O.bf16_round(w[f"l0.mix.{n}.b"] * f)
    w["l0.mix.q.norm"] = O.bf16_round(np.linspace(0.2, 1.5, 16))
    w["l0.mix.k.norm"] = O.bf16_round(np.linspace(1.8, 0.4, 16))
    toks = tokens_for(cfg, 80, seed=3)
    ref = O.forward(cfg, w, toks)
    for n in "qkv":
        assert float(row_errors(O.forward(cfg, dict(w, **{f"l0.mix.{n}.b": w[f"l0.mix.{n}.b"] * 0}), toks), ref).median()) > 0.03, n
    assert float(row_errors(O.forward(cfg, dict(w, **{"l0.mix.q.norm": np.ones(16), "l0.mix.k.norm": np.ones(16)}), toks), ref).median()) > 0.03
    logits_agree(cfg, w, toks, ref, ([80], [33, 2, 20], [1]))


def test_the_output_gate_is_per_channel_and_reads_the_layers_input():
    cfg = config([layer(attn(4, 2, 16, 24, 8), None)], width=64)
    w = O.random_weights(cfg, seed=7)
    w["l0.mix.g"] = O.bf16_round(w["l0.mix.g"] * 4.0)
    toks = tokens_for(cfg, 80, seed=3)
    ref = O.forward(cfg, w, toks)
    coarse = np.repeat(w["l0.mix.g"].reshape(4, 24, 64)[:, :1], 24, axis=1).reshape(96, 64)
    assert float(row_errors(O.forward(cfg, dict(w, **{"l0.mix.g": coarse}), toks), ref).median()) > 0.05
    logits_agree(cfg, w, toks, ref, ([80], [33, 2, 20], [1]))


def test_the_dense_unit_is_the_tanh_form_of_gelu():
    """Gate values around the two forms' largest difference and a large second factor: the erf form is several tolerances away."""
    cfg = config([layer(AT_ONE, {"kind": "dense", "ff": 32})], width=32)
    w = O.random_weights(cfg, seed=8)
    w["l0.mix.o"] = O.bf16_round(w["l0.mix.o"] * 0.01)
    w["l0.mlp.gate"] = O.bf16_round(w["l0.mlp.gate"] * 2.2)
    w["l0.mlp.up"] = O.bf16_round(w["l0.mlp.up"] * 20.0)
    toks = tokens_for(cfg, 60, seed=3)
    x = O.embedding(cfg, w, toks)
    u = O.rms_norm(x, w["l0.norm1"], 1e-5)
    p = O.layer_params(w, 0, "mlp")
    z = u @ p["gate"].T
    erf = 0.5 * z * (1.0 + np.vectorize(math.erf)(z / math.sqrt(2.0)))
    y = x + O.attention(u, O.layer_params(w, 0, "mix"), cfg["layers"][0]["mixer"], 1e-5)
    right, wrong = y + O.dense_ff(u, p), y + (erf * (u @ p["up"].T)) @ p["down"].T
    assert float(row_errors(wrong, right).median()) > 1e-4
    model, _ = build(cfg, torch.float32, weights=w)
    _, hidden = model.forward(torch.tensor([toks]), output_hidden_states=True)
    assert err(hidden[0, 0], right) < 1e-5


# ----------------------------------------------------------------------------------------------------------- router and experts
def route_variant(cfg, w, toks, fn):
    """The oracle's logits with its router replaced by fn(scores, correction, router) -> [(index, weight), ...] per row."""
    keep = O.route

    def route(h, router_w, correction, r):
        z = h @ router_w.T
        s = np.exp(z - z.max(-1, keepdims=True))
        s = s / s.sum(-1, keepdims=True)
        pairs = [fn(row, np.asarray(correction, np.float64), r) for row in s]
        return [[e for e, _ in p] for p in pairs], [[g for _, g in p] for p in pairs]

    O.route = route
    try:
        return O.forward(cfg, w, toks)
    finally:
        O.route = keep


def choose(s, c, r, choice=None, group=None, mask=-np.inf, weight=None, total=None):
    n, per = len(s), len(s) // r["groups"]["count"]
    choice = s + c if choice is None else choice(s, c)
    gs = (group or (lambda v: v.max(-1)))(choice.reshape(-1, per))
    alive = np.argsort(-gs, kind="stable")[:r["groups"]["keep"]]
    cand = np.where(np.isin(np.arange(n) // per, alive), choice, mask)
    top = np.argsort(-cand, kind="stable")[:r["top"]]
    w = s[top] if weight is None else weight(s, c)[top]
    return list(zip(top.tolist(), (w / (w.sum() if total is None else total)).tolist()))


ROUTED = moe(9, 3, 24, identity=3, groups=(4, 2), limit=1.0)


def routed_model(shift=0.0, seed=11):
    cfg = config([layer(AT_ONE, ROUTED)], width=64, vocab=200)
    w = O.random_weights(cfg, seed=seed)
    w["l0.mix.o"] = O.bf16_round(w["l0.mix.o"] * 0.1)
    w["l0.mlp.correction"] = O.bf16_round(w["l0.mlp.correction"] * 2.0 + shift)
    for n in w:
        if n.endswith(".down"):
            w[n] = O.bf16_round(w[n] * 2.0)
    return cfg, w, tokens_for(cfg, 130, seed=4)


VARIANTS = {
    "choice without correction": lambda s, c, r: choose(s, c, r, choice=lambda s, c: s),
    "groups scored without correction": lambda s, c, r: choose(s, c, r, group=lambda v: (v - c.reshape(v.shape)).max(-1)),
    "groups scored by their two best": lambda s, c, r: choose(s, c, r, group=lambda v: np.sort(v, -1)[:, -2:].sum(-1)),
    "weights with correction": lambda s, c, r: choose(s, c, r, weight=lambda s, c: s + c),
    "weights not normalised": lambda s, c, r: choose(s, c, r, total=1.0),
    "identity experts give nothing": lambda s, c, r: [(e, 0.0 if e >= 9 else g) for e, g in choose(s, c, r)],
    "scores over the experts alone": lambda s, c, r: choose(np.where(np.arange(12) < 9, s, 0.0) / s[:9].sum(), c, r),
}


def test_routing_rules_show():
    """Premise for every rule: an oracle that breaks it alone is far away from many rows. The engine agrees with the right one in a prompt on
    either expert path (grouped and tensor-core products), in portions and in decode steps."""
    cfg, w, toks = routed_model()
    ref = O.forward(cfg, w, toks)
    assert np.allclose(route_variant(cfg, w, toks, choose), ref)
    for name, fn in VARIANTS.items():
        moved = row_errors(route_variant(cfg, w, toks, fn), ref)
        assert int((moved > 0.02).sum()) >= 12, name
    logits_agree(cfg, w, toks, ref, ([130], [64, 2, 9, 8, 7], [40, 3] + [2] * 20, [1]))


def test_dropped_groups_lose_even_to_negative_choice_scores():
    """Corrections that push every choice score below zero: counting the dropped groups' experts as 0 instead of out of reach would choose
    them first."""
    cfg, w, toks = routed_model(shift=-1.5)
    ref = O.forward(cfg, w, toks)
    zeroed = route_variant(cfg, w, toks, lambda s, c, r: choose(s, c, r, mask=0.0))
    assert float(row_errors(zeroed, ref).median()) > 0.05
    logits_agree(cfg, w, toks, ref, ([130], [64, 2, 9, 8, 7], [1]))


def test_the_experts_bounds_show():
    """Expert inputs large enough that both bounds bite on both sides. Premise: an oracle without the bounds, with the gate bounded below
    too, with the second factor bounded on one side only, without the shift by one, or with slope 1 is far away."""
    cfg, w, toks = routed_model(seed=12)
    for n in w:
        if n.endswith(".gate") or n.endswith(".up"):
            w[n] = O.bf16_round(w[n] * 1.5)
    ref = O.forward(cfg, w, toks)
    keep = O.expert

    def variant(act):
        O.expert = lambda h, gate, up, down, limit: act(h @ gate.T, h @ up.T, limit) @ down.T
        try:
            return O.forward(cfg, w, toks)
        finally:
            O.expert = keep

    unit = lambda g, u, slope=1.702, one=1.0: g * O.sigmoid(slope * g) * (u + one)  # noqa: E731
    assert np.allclose(variant(lambda g, u, m: unit(np.minimum(g, m), np.clip(u, -m, m))), ref)
    for act in (lambda g, u, m: unit(g, u), lambda g, u, m: unit(np.clip(g, -m, m), np.clip(u, -m, m)), lambda g, u, m: unit(np.minimum(g, m), np.minimum(u, m)),
                lambda g, u, m: unit(np.minimum(g, m), np.maximum(u, -m)), lambda g, u, m: unit(np.minimum(g, m), np.clip(u, -m, m), one=0.0),
                lambda g, u, m: unit(np.minimum(g, m), np.clip(u, -m, m), slope=1.0)):
        assert float(row_errors(variant(act), ref).median()) > 0.01
    logits_agree(cfg, w, toks, ref, ([130], [64, 2, 9, 8, 7], [1]))


def test_a_tokens_experts_do_not_depend_on_the_rest_of_the_portion():
    """The same tokens at the end of portions of every length around the limits between the expert paths (8 / 9 and 63 / 64 rows)."""
    cfg, w, toks = routed_model(seed=13)
    ref = O.forward(cfg, w, toks)
    for dtype in (torch.float32, torch.bfloat16):
        model, _ = build(cfg, dtype, weights=w)
        eng = model._ensure_engine()
        kv = eng.new_kv(1, 256)
        for n in (2, 7, 8, 9, 10, 63, 64, 65, 127, 128, 129):
            assert close(run_schedule(eng, kv, 0, toks, [130 - n, n]), ref, dtype), n


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
    """Prompts of one, two and three tokens, alone and continued one by one."""
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
def test_long_decoding(dtype):
    cfg = CFG_MAIN
    model, w = build(cfg, dtype)
    eng = model._ensure_engine()
    kv = eng.new_kv(2, 256)
    toks = tokens_for(cfg, 170, seed=5)
    got = run_schedule(eng, kv, 0, toks, [8])          # 162 decode steps: most keys are decoded ones
    ref = O.forward(cfg, w, toks)
    assert close(got[-40:], ref[-40:], dtype)
    assert close(got, ref, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cfg", [CFG_MAIN, CFG_TILE], ids=["main", "tile"])
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
    run_schedule(eng, kv, 0, a, [50])                      # leaves cache rows of a longer request behind
    kv.free_slot(0)
    assert kv.lengths(2)[0] == 0
    again = run_schedule(eng, kv, 0, b, [20])
    assert err(again, fresh) < 1e-6
    third = run_schedule(eng, kv, 0, b, [2, 2])            # restart on a slot that was not freed, shortest portions
    assert err(third, fresh) < 2e-5
    with pytest.raises(ValueError):
        eng.append_tokens(kv, 0, [0] * 300, [], restart=False)   # beyond the slot's capacity


def test_every_pass_of_a_looped_layer_has_its_own_cache():
    """Three passes over both layers against an oracle that runs six layers with the same tensors and nothing in between: equal only if
    no pass shares a cache with another, in a prompt, in portions and in decode steps. Premise: one pass less is far away."""
    cfg = CFG_ONE
    w = O.random_weights(cfg, seed=0)
    toks = tokens_for(cfg, 60, seed=6)
    ref = O.forward(cfg, w, toks)
    x = O.embedding(cfg, w, toks)
    for _ in range(3):
        for i in range(2):
            x = O.layer_step(x, w, i, cfg["layers"][i], cfg["norm"]["eps"])
    assert np.allclose(ref, O.rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ np.asarray(w["embed"], np.float64).T)
    assert float(row_errors(O.forward(dict(cfg, loop=dict(cfg["loop"], times=2)), w, toks), ref).median()) > 0.05
    logits_agree(cfg, w, toks, ref, ([60], [13, 2, 20], [2]))


# ----------------------------------------------------------------------------------------------------------- edges
def sharp_model(seed=7, factor=None, base=50.0):
    """One attention layer whose score factor is scaled up until the softmax is almost an argmax: for most positions ONE visible key
    carries the output, as often one of the first as any other. A key too many or too few (at the row's own position, the edge of a key
    tile of 32, a key split, a portion) then moves many rows by far more than the tolerance."""
    cfg = config([layer(attn(4, 2, 16, 16, 8, base=base, factor=factor, scale=3.0), None)], width=48, vocab=400)
    w = O.random_weights(cfg, seed=seed)
    for n in "qk":
        w[f"l0.mix.{n}.b"] = O.bf16_round(w[f"l0.mix.{n}.b"] * 0.2)
    w["l0.mix.v"] = O.bf16_round(w["l0.mix.v"] * 3.0)
    return cfg, w


def masked_oracle(cfg, w, toks, sees):
    """The oracle's logits for one attention layer whose row i sees the positions j with sees(i, j)."""
    eps, p, mix = cfg["norm"]["eps"], O.layer_params(w, 0, "mix"), cfg["layers"][0]["mixer"]
    x = O.embedding(cfg, w, toks)
    u = O.rms_norm(x, w["l0.norm1"], eps)
    q, k, v = O.queries_keys_values(u, p, mix, eps)
    per = mix["heads"] // mix["kv_heads"]
    out = np.zeros((len(toks), mix["heads"], mix["vdim"]))
    for i in range(len(toks)):
        js = [j for j in range(i + 1) if sees(i, j)]
        for a in range(mix["heads"]):
            if js:
                out[i, a] = O.softmax_attend(k[js, a // per] @ q[i, a] * mix["scale"], v[js, a // per])
    x = x + (out.reshape(len(toks), -1) * O.sigmoid(u @ p["g"].T)) @ p["o"].T
    return O.rms_norm(x, w["final.norm"], eps) @ np.asarray(w["embed"], np.float64).T


def test_every_visible_key_counts_near_and_far():
    T = 420
    cfg, w = sharp_model()
    toks = tokens_for(cfg, T, seed=9)
    ref = O.forward(cfg, w, toks)
    assert np.allclose(masked_oracle(cfg, w, toks, lambda i, j: True), ref)
    # the test's premise: a row that loses its own key, the first key, the keys at the edges of tiles of 32, or the far ones changes
    for name, sees, rows in (("own", lambda i, j: j < i, 20), ("first", lambda i, j: j > 0, 3), ("tile edges", lambda i, j: j % 32 not in (0, 31), 60),
                             ("far", lambda i, j: i - j < 200, 60)):
        assert int((row_errors(masked_oracle(cfg, w, toks, sees), ref) > 2e-2).sum()) >= rows, name
    model, _ = build(cfg, torch.float32, weights=w, max_batch=2, max_seq=1024, max_rows=512)
    eng = model._ensure_engine()
    kv = eng.new_kv(2, 1024)
    assert err(run_schedule(eng, kv, 0, toks, [T]), ref) < 2e-4, "whole prompt"
    assert err(run_schedule(eng, kv, 1, toks, [31, 2, 33, 64, 1, 5, 2, 2, 130]), ref) < 2e-4, "portions that end at and around tile edges, then decode steps"
    assert err(run_schedule(eng, kv, 0, toks, [32, 32, 31, 1, 2, 200]), ref) < 2e-4, "portions of whole tiles"
    assert err(run_schedule(eng, kv, 1, toks, [300]), ref) < 2e-4, "120 decode steps over split keys"
    assert err(run_schedule(eng, kv, 1, toks, [2]), ref) < 2e-4, "decode steps from the second position on"


def test_positions_far_along_keep_their_angles_and_their_scaling():
    """Rotations at positions in the thousands (angles of hundreds to thousands of radians at the fastest pair), slowed down and plain.
    Premise: a scaling factor that is a little off, or applied twice, is far away there."""
    T = 2200
    cfg, w = sharp_model(seed=21, factor=6.0, base=20.0)
    cfg["layers"].append(copy.deepcopy(cfg["layers"][0]))
    del cfg["layers"][1]["mixer"]["rot"]["scaling"]
    w = dict(O.random_weights(cfg, seed=22), **w)
    toks = tokens_for(cfg, T, seed=41)
    ref = O.forward(cfg, w, toks)[-40:]
    for factor in (6.05, 36.0, 1.0):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["rot"]["scaling"]["factor"] = factor
        assert int((row_errors(O.forward(other, w, toks)[-40:], ref) > 2e-2).sum()) >= 20, factor
    model, _ = build(cfg, torch.float32, weights=w, max_seq=2304, max_rows=2304, max_batch=1)
    eng = model._ensure_engine()
    kv = eng.new_kv(1, 2304)
    got = run_schedule(eng, kv, 0, toks, [2190])
    assert err(got[-40:], ref) < 5e-4          # scores of tens, angles of thousands: their fp32 rounding is a few 1e-6 each


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
    out = model.generate(prompts, max_new_tokens=24)
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
    for cfg, names in ((CFG_ODD, ("l0.mlp.correction", "l0.mlp.e6.down", "l1.mix.k.b", "l2.mix.v.b", "l1.mlp.gate", "embed.norm")), (CFG_MAIN, ("l1.mix.q.norm", "l3.mix.g"))):
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

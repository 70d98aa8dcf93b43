"""The plain statement of the Lakadra design (tests/plain_lakadra.py) against closed forms, the faults it must show, and
the host side of the library for this design (configuration, parameter names, cache planes and states, random weights):
everything here runs without a GPU."""
import copy
import json
import math

import numpy as np
import pytest

import lakadra_cases as lc
import plain_lakadra as pl
from helpers import TOL_F32, random_tokens


# ---- the plain mechanisms against closed forms -----------------------------------------------------------
def test_a_lightning_state_is_a_decayed_sum_over_the_past():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((9, 4)), rng.standard_normal((9, 4)), rng.standard_normal((9, 3))
    o = pl.lightning_state(q, k, v, 0.7)
    for t in range(9):
        assert np.allclose(o[t], sum(0.7 ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1)))
    assert np.allclose(pl.lightning_state(q, k, v, 0.0), (q * k).sum(1, keepdims=True) * v)  # nothing is kept


def test_norms_with_a_gain_around_zero_and_around_one():
    x = np.array([[3.0, -4.0]])
    r = math.sqrt(12.5 + 1e-3)
    assert np.allclose(pl.unit_rms(x, 1e-3), x / r) and np.allclose(pl.layer_norm_of(x, np.array([0.0, 1.0]), 1e-3), x / r * [1, 2])


def test_rotated_scores_depend_on_the_distance_only_in_both_pairings():
    rng = np.random.default_rng(1)
    for pairing in ("neighbours", "halves"):
        q, k = np.tile(rng.standard_normal(10), (30, 1)), np.tile(rng.standard_normal(10), (30, 1))
        a, b = pl.turned(q, 100.0, 8, pairing, 2.0), pl.turned(k, 100.0, 8, pairing, 2.0)
        assert np.allclose(a[9] @ b[4], a[25] @ b[20]) and not np.allclose(a[9] @ b[4], a[9] @ b[3])
        assert np.allclose(a[:, 8:], q[:, 8:])  # numbers beyond the rotated part pass
    x = np.zeros((4, 8))
    x[:, 1] = 1.0
    angle = 3 * 100.0 ** (-2.0 / 8) / 2.0
    y = pl.turned(x, 100.0, 8, "halves", 2.0)[3]
    assert np.allclose(y[[1, 5]], [math.cos(angle), math.sin(angle)]) and np.allclose(np.delete(y, [1, 5]), 0)
    y = pl.turned(x, 100.0, 8, "neighbours")[3]
    assert np.allclose(y[[0, 1]], [-math.sin(3.0), math.cos(3.0)]) and np.allclose(y[2:], 0)


def test_one_added_to_the_denominator_takes_weight_and_gives_nothing_back():
    s, v = np.array([[0.3, -1.0, 2.0]]), np.eye(3)
    seen = np.array([[True, True, False]])
    e = np.exp(s[0, :2])
    assert np.allclose(pl.weighted_values(s, seen, v, added=1.0)[0], [*(e / (1 + e.sum())), 0])
    assert np.allclose(pl.weighted_values(s, seen, v)[0], [*(e / e.sum()), 0])
    assert np.allclose(pl.weighted_values(s - 800, seen, v, added=1.0), 0) and np.allclose(pl.weighted_values(s + 800, seen, v, added=1.0).sum(), 1)


def test_a_convolution_looks_back_only_and_ends_on_the_current_token():
    x = np.zeros((6, 2))
    x[2] = [1.0, 10.0]
    y = pl.causal_convolution(x, np.array([[0.1, 0.2, 0.3], [1.0, 2.0, 3.0]]), np.array([0.0, 5.0]))
    assert np.allclose(y[:, 0], [0, 0, 0.3, 0.2, 0.1, 0]) and np.allclose(y[:, 1], [5, 5, 35, 25, 15, 5])


def test_the_gated_recurrence_forgets_by_its_gates_and_starts_from_zero():
    T, B, P = 5, 2, 3
    u = np.random.default_rng(2).standard_normal((T, B * P))
    zero, off = np.zeros((B, P, P)), np.full((B, P), -800.0)
    S = pl.gated_linear_states(u, zero, off, zero, -off, np.zeros(B * P))
    assert np.allclose(S, 0)  # r = 0: the decay is one and nothing enters
    S = pl.gated_linear_states(u, zero, -off, zero, np.zeros((B, P)), np.full(B * P, 5.0))
    assert np.allclose(S, 0.5 * u, atol=1e-9)  # r = 1 and a large lam: all is forgotten at once, i = 1/2
    ra = np.random.default_rng(3).standard_normal((B, P, P))
    S = pl.gated_linear_states(u, ra, np.zeros((B, P)), zero, -off, np.full(B * P, -3.0))
    a = np.exp(-8 * pl.sigmoid(np.concatenate([ra[b] @ u[1, b * P: (b + 1) * P] for b in range(B)])) * math.log1p(math.exp(-3.0)))
    assert np.allclose(S[1], a * S[0] + np.sqrt(1 - a * a) * u[1])


def test_experts_are_chosen_by_corrected_scores_within_the_best_groups_and_weighed_without():
    z = np.log(np.array([[0.4, 0.1, 0.3, 0.2, 0.05, 0.05]]) / 1.1)
    ids, w = pl.choose_experts(z, np.zeros(6), 2, 1, 1)
    assert ids.tolist() == [[0, 2]] and np.allclose(w * 1.1, [[0.4, 0.3]])
    c = np.array([-0.5, 0.0, -0.9, -0.9, 0.0, 0.2])
    ids, w = pl.choose_experts(z, c, 2, 3, 1)  # groups {0, 1}, {2, 3}, {4, 5}: the last one holds the largest corrected score
    assert ids.tolist() == [[5, 4]] and np.allclose(w * 1.1, [[0.05, 0.05]])
    ids, w = pl.choose_experts(z, c - 3.0, 3, 3, 2)  # all choice scores negative: an expert of the group left out does not come back
    assert ids.tolist() == [[5, 1, 4]]


def test_identity_experts_hand_on_the_input_and_the_shared_expert_has_a_gate():
    h = np.array([[1.0, -2.0]])
    mlp = lc.moe(1, 1, 2, 1, 1, 1, 1)
    w = {"router": np.zeros((2, 2)), "correction": np.zeros(2), "e0.up": np.array([[2.0, 0.0]]), "e0.down": np.array([[1.0], [3.0]]),
         "shared.up": np.array([[0.0, -1.0]]), "shared.down": np.array([[1.0], [0.0]]), "shared.sg": np.array([[0.0, 0.0]])}
    assert np.allclose(pl.experts(h, w, "", mlp), 0.5 * h + 0.5 * np.array([[4.0, 12.0]]) + 0.5 * np.array([[4.0, 0.0]]))
    assert np.allclose(pl.squared_relu_unit(np.array([[-3.0, 0.0]]), w["e0.up"], w["e0.down"]), 0)


# ---- faults must show --------------------------------------------------------------------------------------
def _faults(cfg):
    """(name, changed configuration, function that changes the weights) for every constant and tensor kind."""
    out = []

    def cfg_fault(name, fn):
        c = copy.deepcopy(cfg)
        fn(c)
        out.append((name, c, None))

    def w_fault(name, tensor, fn):
        out.append((name, cfg, lambda w: {**w, tensor: fn(w[tensor])}))

    zero, flip = lambda a: a * 0, lambda a: a[:, ::-1].copy()
    cfg_fault("logit scale", lambda c: c.update(logit_scale=c["logit_scale"] * 1.3))
    cfg_fault("soft cap", lambda c: c.update(logit_softcap=c["logit_softcap"] * 0.5))
    cfg_fault("eps", lambda c: c["norm"].update(eps=0.5))
    w_fault("final norm's gain", "final.norm", zero)
    for i, layer in enumerate(cfg["layers"]):
        m, kind, p, at = layer["mixer"], layer["type"], f"l{i}.mix.", f"layer {i}: "
        mixer = lambda c, i=i: c["layers"][i]["mixer"]
        w_fault(at + "norm's gain", f"l{i}.norm1", zero)
        if kind == "lightning":
            cfg_fault(at + "decays in another order", lambda c: mixer(c)["decay"].reverse())
            cfg_fault(at + "a state that is forgotten", lambda c: mixer(c).update(decay=[0.0] * m["heads"]))
            w_fault(at + "gate", p + "g", lambda a: -a)
            w_fault(at + "gain", p + "norm", lambda a: a * 0 + 1)
        elif kind == "latent_attention":
            cfg_fault(at + "scale", lambda c: mixer(c).update(scale=m["scale"] * 2))
            if m.get("kv_from") is None:
                cfg_fault(at + "rotary base", lambda c: [l["mixer"]["rot"].update(base=m["rot"]["base"] * 20) for l in c["layers"]
                                                         if l["type"] == kind and l["mixer"]["rot"] == m["rot"]])
                w_fault(at + "latent norm's gain", p + "dkv.norm", lambda a: a * 0 + 1)
            w_fault(at + "query norm's gain", p + "dq.norm", lambda a: a * 0 + 1)
            w_fault(at + "rotated queries", p + "uq", lambda a: np.where((np.arange(len(a)) % (m["dim"] + m["rot_dim"]) < m["dim"])[:, None], a, 0))
        else:
            a_, b_ = m["left"], m["right"]
            cfg_fault(at + "left's factor", lambda c: mixer(c).update(left_scale=m["left_scale"] * 0.5))
            cfg_fault(at + "right's factor", lambda c: mixer(c).update(right_scale=m["right_scale"] * 0.5))
            cfg_fault(at + "window", lambda c: mixer(c)["left"]["mask"].update(size=a_["mask"]["size"] // 2 + 1 if a_["mask"]["size"] > 1 else 2))
            cfg_fault(at + "scale", lambda c: mixer(c)["left"].update(scale=a_["scale"] * 2))
            if a_["mask"]["size"] > 1:  # a token that sees itself only has no distances
                if a_["rot"]["dims"] > 2:  # one pair turns by the position itself, whatever the base
                    cfg_fault(at + "rotary base", lambda c: mixer(c)["left"]["rot"].update(base=2.0))
                cfg_fault(at + "slower rotation", lambda c: mixer(c)["left"]["rot"].update(scaling={"factor": 40.0}))
            for n in "qkvo":
                if n != "k" or a_["mask"]["size"] > 1:
                    w_fault(f"{at}bias of {n}", f"{p}left.{n}.b", zero)
            w_fault(at + "gates per head", p + "left.g", lambda a: -a)
            for n in ("y.b", "x.b", "conv.b", "ra.b", "ri.b"):
                w_fault(f"{at}{n}", f"{p}right.{n}", zero)
            w_fault(at + "lam", p + "right.lam", lambda a: a + 1.5)
            w_fault(at + "gates' matrix the wrong way round", p + "right.ri", lambda a: a.transpose(0, 2, 1).copy())
            w_fault(at + "decay gates", p + "right.ra", lambda a: a * -2)
            if b_["conv"] > 1:
                w_fault(at + "convolution turned round", p + "right.conv", flip)
        mlp = layer.get("mlp")
        if mlp:
            q = f"l{i}.mlp."
            w_fault(at + "shared expert's gate", q + "shared.sg", lambda a: -a)
            if mlp["router"]["top"] < mlp["router"]["experts"] + mlp["router"]["identity"]:
                w_fault(at + "corrections", q + "correction", lambda a: a[::-1].copy())
    return out


@pytest.mark.parametrize("case", sorted(lc.CASES))
def test_every_constant_and_tensor_kind_moves_the_logits(case):
    """Every fault moves the float32 models' logits by more than thirty times what they may differ, and nearly every one by
    more than a bfloat16 engine may (tests/test_lakadra_gpu.py: no position beyond three times the largest gap that rounding
    the stored activations opens, at most a fifth of the positions beyond three times the gap's 80th percentile)."""
    cfg = lc.CASES[case]
    toks = random_tokens(5, 150, cfg["vocab"])
    sharp, calm = (lc.draw_weights(cfg, 26, calm=c) for c in (False, True))
    ref = {id(w): pl.forward(toks, w, cfg) for w in (sharp, calm)}
    gap = np.abs(pl.forward(toks, calm, cfg, r=pl.to_bf16) - ref[id(calm)]).max(axis=1)
    faults = _faults(cfg)
    assert len(faults) >= 35
    missed, faint = [], []
    for name, c, change in faults:
        move = lambda w: np.abs(pl.forward(toks, change(w) if change else w, c) - ref[id(w)]).max(axis=1)
        if not move(sharp).max() > 30 * TOL_F32 * np.abs(ref[id(sharp)]).max():
            missed.append(name)
        err = move(calm)
        if not (err.max() > 3.0 * gap.max() or int((err > 3.0 * np.percentile(gap, 80)).sum()) > len(toks) // 5):
            faint.append(name)
    assert not missed, f"case {case}: no more than single precision may: {missed}"
    assert len(faint) <= len(faults) // 6, f"case {case}: no more than rounding may: {faint}"


@pytest.mark.parametrize("case", sorted(lc.CASES))
def test_what_a_sequence_carries_reaches_far_on(case):
    """The first token shows in the logits a hundred tokens later (a state or a cache that loses its start would not go
    unseen in single precision)."""
    cfg = lc.CASES[case]
    w = lc.draw_weights(cfg, 26)
    toks = random_tokens(6, 140, cfg["vocab"])
    other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    ref = pl.forward(toks, w, cfg)
    far = np.abs(ref - pl.forward(other, w, cfg)).max(axis=1)[100:]
    assert far.min() > 1e-4 * np.abs(ref).max()


# ---- the library's host side ---------------------------------------------------------------------------
def _spec(cfg):
    from bitnet_c_b200.config import architecture_of
    arch = architecture_of(cfg)
    return arch, arch.to_spec(arch.read_config(cfg))


def test_the_configuration_becomes_blocks_and_the_designs_tensor_names():
    from bitnet_c_b200.engine.model import parameter_table
    for name, cfg in lc.CASES.items():
        arch, spec = _spec(cfg)
        assert arch.name == "Lakadra" and len(spec.blocks) == len(spec.schedule) == len(cfg["layers"]) and not spec.tie_embeddings
        names = {arch.tensor_name(p): tuple(s.shape) for p, s in parameter_table(spec).items()}
        assert names == {n: tuple(s) for n, s in lc.tensor_shapes(cfg).items()}, name
        assert not any(s.integer or s.optional for s in parameter_table(spec).values())
        assert arch.config_to_dict(arch.read_config(cfg)) == cfg


def test_parts_carry_every_constant_of_the_configuration():
    _arch, spec = _spec(lc.CASE_A)
    assert (spec.head.scale, spec.head.softcap, spec.final_norm.eps, spec.final_norm.one_plus) == (0.7, 12.0, 1e-5, True)
    assert [e.cache_of for e in spec.schedule] == [None, None, None, 0, None, None, None, 4]
    lat, pair, light, reader = (spec.blocks[i].mixer for i in range(4))
    assert (lat.n_heads, lat.head_dim, lat.rot_dim, lat.v_head_dim, lat.q_rank, lat.kv_rank, lat.scale, lat.window) == (3, 16, 8, 20, 40, 24, 0.5, 0)
    assert (lat.position.dims, lat.position.base, lat.position.pairing, lat.position.slowdown) == (8, 300.0, "neighbours", 1.0)
    assert lat.own_kv and not reader.own_kv and not lat.head_gate and not lat.sink and (reader.q_rank, reader.scale) == (24, 0.7)
    a, b = pair.left, pair.right
    assert (pair.left_scale, pair.right_scale) == (0.8, 1.1)
    assert (a.n_heads, a.n_kv_heads, a.head_dim, a.v_head_dim, a.window, a.scale) == (6, 2, 16, 24, 37, 0.4)
    assert (a.position.dims, a.position.base, a.position.pairing, a.position.slowdown) == (8, 1000.0, "halves", 3.0)
    assert a.zero_sink and a.head_gate and a.proj_bias and a.out_bias and not a.sink
    assert spec.blocks[5].mixer.left.position.slowdown == 1.0 and spec.blocks[5].mixer.left_scale == -0.6
    assert (b.inner, b.parts, b.conv_taps) == (48, 4, 3)
    assert (light.n_heads, light.head_dim, light.v_head_dim, light.decay, light.norm_eps) == (3, 12, 20, (0.7, 0.97, 0.9995), 1e-5)
    assert spec.blocks[2].ffn is None
    moe = spec.blocks[1].ffn
    assert (moe.n_experts, moe.identity, moe.top, moe.groups, moe.keep_groups, moe.expert_ff, moe.shared_ff) == (4, 4, 3, 2, 1, 16, 24)
    assert moe.correction and moe.shared_gate and moe.scores == "softmax" and not moe.renormalise and moe.activation == "relu2"


def test_groups_identity_experts_and_a_shared_expert_may_be_left_out():
    cfg = copy.deepcopy(lc.CASE_B)
    mlp = cfg["layers"][0]["mlp"]
    mlp["router"] = {"experts": 4, "top": 2}
    mlp["shared"] = None
    cfg.pop("logit_softcap")
    _arch, spec = _spec(cfg)
    moe = spec.blocks[0].ffn
    assert (moe.identity, moe.groups, moe.keep_groups, moe.shared_ff, moe.shared_gate, spec.head.softcap) == (0, 1, 1, 0, False, 0.0)


def _mix(c, i):
    return c["layers"][i]["mixer"]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: _mix(c, 1)["left"].update(heads=5), "multiple"),
    (lambda c: _mix(c, 1)["left"]["rot"].update(dims=7), "rot"),
    (lambda c: _mix(c, 1)["left"]["rot"].update(dims=18), "rot"),
    (lambda c: _mix(c, 1)["left"]["rot"].update(scaling={"factor": 0}), "factor"),
    (lambda c: _mix(c, 1)["left"].pop("mask"), "mask"),
    (lambda c: _mix(c, 1)["right"].update(blocks=5), "multiple"),
    (lambda c: _mix(c, 1)["right"].update(conv=17), "conv"),
    (lambda c: _mix(c, 1).pop("left_scale"), "left_scale"),
    (lambda c: _mix(c, 2).update(decay=[0.5, 0.5]), "decay"),
    (lambda c: _mix(c, 2).update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda c: _mix(c, 0)["rot"].update(dims=6), "rot_dim"),
    (lambda c: _mix(c, 0).pop("q_rank"), "q_rank"),
    (lambda c: _mix(c, 3).update(kv_from=1), "kv_from"),
    (lambda c: _mix(c, 3).update(kv_from=3), "kv_from"),
    (lambda c: _mix(c, 7).update(kv_from=3), "kv_from"),
    (lambda c: _mix(c, 3).update(kv_rank=32), "kv_rank"),
    (lambda c: _mix(c, 3)["rot"].update(base=7.0), "rot"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.update(logit_softcap=-1), "logit_softcap"),
    (lambda c: c.pop("vocab"), "vocab"),
])
def test_configurations_that_cannot_be_built_are_refused_by_name(change, message):
    from bitnet_c_b200.config import ConfigError, architecture_of
    cfg = copy.deepcopy(lc.CASE_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        architecture_of(cfg).read_config(cfg)


def test_planes_and_states_are_what_the_layers_ask_for():
    import torch
    from bitnet_c_b200.csrc import ops
    from bitnet_c_b200.engine import Model
    _arch, spec = _spec(lc.CASE_A)
    cache = Model(spec, dtype="bfloat16", device=None).new_cache(max_tokens=64 * 8, max_seqs=2, allocate=False)
    groups = {(g.request.n_kv_heads, g.request.head_dim, g.request.window, g.request.values_in_keys): g.entries for g in cache.groups}
    assert groups == {(1, 32, 0, True): [0], (1, 64, 0, True): [4], (2, 16, 37, False): [1], (4, 32, 100, False): [5]}
    want = {(1, "right"): ops.gated_linear_floats(48, 3), (5, "right"): ops.gated_linear_floats(96, 5),
            2: ops.gated_state_floats(3, 3, 12, 20, 1), 6: ops.gated_state_floats(4, 4, 32, 16, 1)}
    assert {k: r.shape for k, r in cache.state_requests.items()} == {k: (n,) for k, n in want.items()}
    assert all(r.dtype == torch.float32 for r in cache.state_requests.values())
    assert ops.gated_linear_floats(48, 3) == 4 * 48 and ops.gated_linear_floats(35, 1) == 36


def test_slowed_down_frequencies_are_the_plain_ones_over_the_factor():
    from bitnet_c_b200.config import RotaryBlendSpec
    from bitnet_c_b200.parts.position import blended_frequencies
    plain, slow = (blended_frequencies(RotaryBlendSpec(dims=12, base=500.0, slowdown=s), wide=True) for s in (1.0, 8.0))
    assert np.allclose(plain[0], 500.0 ** (-np.arange(6) / 6.0)) and np.allclose(slow[0] * 8.0, plain[0]) and slow[1] == plain[1] == 1.0


def test_random_weights_of_the_design_have_its_tensors_only(tmp_path):
    import bitnet_c_b200 as bn
    from bitnet_c_b200.weights.safetensors_io import SafetensorsFile
    folder = bn.write_random_model(str(tmp_path / "m"), lc.CASE_A, seed=5)
    f = SafetensorsFile(str(tmp_path / "m" / "model.safetensors"))
    try:
        assert {n: tuple(f.entries[n].shape) for n in f.names()} == {n: tuple(s) for n, s in lc.tensor_shapes(lc.CASE_A).items()}
        assert abs(float(f.read("l0.norm1").float().mean())) < 0.1
    finally:
        f.close()
    assert json.load(open(tmp_path / "m" / "config.json"))["architecture"] == "Lakadra" and folder

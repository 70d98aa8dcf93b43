"""The plain statement of the Rudolix design (tests/plain_rudolix.py) against closed forms, the faults it must show, and
the host side of the library for this design (configuration, parameter names, states by name, random weights):
everything here runs without a GPU."""
import copy
import json
import math

import numpy as np
import pytest

import plain_rudolix as pr
import rudolix_cases as rc
from helpers import TOL_F32, random_tokens


# ---- the plain mechanisms against closed forms -----------------------------------------------------------
def test_a_layer_norm_takes_mean_and_scale_away():
    rng = np.random.default_rng(0)
    x = rng.standard_normal((5, 12)) * 7 + 3
    y = pr.layer_norm(x, 1.0, 0.0, 1e-12)
    assert np.allclose(y.mean(1), 0) and np.allclose((y * y).mean(1), 1)
    assert np.allclose(pr.layer_norm(x, 2.0, -1.0, 1e-12), 2 * y - 1)
    assert np.allclose(pr.layer_norm(np.full((1, 4), 9.0), 1.0, 0.5, 1e-5), 0.5)  # eps keeps a constant row finite


def test_a_causal_convolution_looks_back_only_and_ends_on_the_current_token():
    x = np.zeros((6, 2))
    x[2] = [1.0, 10.0]
    taps = np.array([[0.1, 0.2, 0.3], [1.0, 2.0, 3.0]])
    y = pr.causal_convolution(x, taps)
    assert np.allclose(y[:, 0], [0, 0, 0.3, 0.2, 0.1, 0]) and np.allclose(y[:, 1], [0, 0, 30, 20, 10, 0])
    assert np.allclose(pr.causal_convolution(x, taps[:, 2:]), x * [0.3, 3.0])  # one tap: no memory
    assert np.allclose(pr.causal_convolution(x, taps, np.array([5.0, -5.0])), y + [5.0, -5.0])


def test_streams_are_mixed_from_the_old_ones_and_indexed_from_and_to():
    xs = np.arange(6.0).reshape(3, 1, 2)
    mix = np.zeros((3, 3))
    mix[0, 2] = 1.0  # stream 0 goes to stream 2
    mix[2, 0] = 10.0
    y = np.array([[100.0, 200.0]])
    new = pr.update_streams(xs, mix, np.array([0.0, 1.0, -1.0]), 0.5, y)
    assert np.allclose(new[0], 10 * xs[2]) and np.allclose(new[1], 0.5 * y) and np.allclose(new[2], xs[0] - 0.5 * y)
    assert np.allclose(pr.read_streams(xs, np.array([1.0, 0.0, 2.0])), xs[0] + 2 * xs[2])


def test_the_delta_rule_replaces_what_a_key_held_and_decays_it():
    k = np.array([[1.0, 0.0], [0.0, 1.0], [1.0, 0.0]])
    v = np.array([[3.0], [5.0], [7.0]])
    o, S = pr.delta_rule(k, k, v, np.ones(3), np.ones(3))
    assert np.allclose(o[:, 0], [3, 5, 7]) and np.allclose(S[:, 0], [7, 5])  # the second write replaced the first
    o, S = pr.delta_rule(k, k, v, np.full(3, 0.5), np.array([1.0, 1.0, 0.0]))
    assert np.allclose(S[:, 0], [3 * 0.25, 5 * 0.5]) and np.allclose(o[2], 3 * 0.25)  # beta 0 writes nothing
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 4)), pr.unit_vector(rng.standard_normal((9, 4))), rng.standard_normal((9, 3))
    g, b = rng.uniform(0.5, 1, 9), rng.uniform(0, 1, 9)
    o, _ = pr.delta_rule(q, k, v, g, b)
    S = np.zeros((4, 3))
    for t in range(9):  # the same as one matrix acting on the state
        S = (np.eye(4) - b[t] * np.outer(k[t], k[t])) @ (g[t] * S) + b[t] * np.outer(k[t], v[t])
        assert np.allclose(o[t], S.T @ q[t])


def test_the_state_space_layer_is_a_decayed_sum_with_a_skip():
    rng = np.random.default_rng(2)
    T, N, P = 11, 5, 3
    x, B, C, dt = rng.standard_normal((T, P)), rng.standard_normal((T, N)), rng.standard_normal((T, N)), rng.uniform(0.1, 1, T)
    y, S = pr.state_space(x, B, C, dt, 0.7, 0.3)
    c = np.cumsum(0.7 * dt)
    for t in range(T):
        want = 0.3 * x[t] + sum(math.exp(c[s] - c[t]) * dt[s] * (C[t] @ B[s]) * x[s] for s in range(t + 1))
        assert np.allclose(y[t], want)
    assert np.allclose(S, sum(math.exp(c[s] - c[-1]) * dt[s] * np.outer(B[s], x[s]) for s in range(T)))


def test_heads_share_groups_in_blocks_and_norms_are_taken_part_by_part():
    assert [pr.shared_head(h, 6, 2) for h in range(6)] == [0, 0, 0, 1, 1, 1] and [pr.shared_head(h, 3, 3) for h in range(3)] == [0, 1, 2]
    y = np.array([[3.0, 4.0, 30.0, 40.0]])
    got = pr.grouped_rms(y, 2, 1e-12)
    assert np.allclose(got[0, :2], got[0, 2:]) and np.allclose(got[0, :2], np.array([3, 4]) / math.sqrt(12.5))
    assert not np.allclose(pr.grouped_rms(y, 1, 1e-12)[0, :2], got[0, :2])


def test_rotated_scores_depend_on_the_distance_only_and_pair_the_halves():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    dots = [float(pr.rotate_halves(q, [p + 5], 8, 100.0)[0, 0] @ pr.rotate_halves(k, [p], 8, 100.0)[0, 0]) for p in (0, 9, 200)]
    assert np.allclose(dots, dots[0])
    x = np.zeros((1, 1, 8))
    x[0, 0, 1] = 1.0
    y = pr.rotate_halves(x, [3], 8, 100.0)[0, 0]
    a = 3 * 100.0 ** (-2.0 / 8)
    assert np.allclose(y[[1, 5]], [math.cos(a), math.sin(a)]) and np.allclose(np.delete(y, [1, 5]), 0.0)
    assert np.allclose(pr.rotate_halves(np.ones((1, 1, 10)), [3], 4, 100.0)[0, 0, 4:], 1.0)  # numbers beyond pass


def test_a_sink_takes_weight_and_gives_nothing_back():
    s = np.array([0.3, -1.0, 2.0, -np.inf])
    w = pr.softmax_with_sink(s, 0.0)
    assert np.allclose(w, np.exp(s) / (1.0 + np.exp(s).sum())) and w[3] == 0
    assert np.allclose(pr.softmax_with_sink(s, -1e9), np.exp(s) / np.exp(s).sum())
    assert pr.softmax_with_sink(s, 60.0).sum() < 1e-20
    q, k, v = np.ones((1, 2)), np.ones((1, 2)), np.array([[3.0, -1.0]])
    assert np.allclose(pr.attend(q, k, v, 0.0, 0.0), v / 2.0)


def test_feed_forwards_in_closed_form():
    z = np.array([[1.0, -2.0, 3.0]])
    r = lambda p: math.sqrt(np.mean(np.array([1.0, 2.0, 3.0]) ** (2 * p)))
    want = 2 * z / r(1) + 3 * z ** 2 / r(2) - z ** 3 / r(3) + 0.5
    assert np.allclose(pr.poly_norm(z, [2, 3, -1, 0.5], 1e-14), want)
    assert np.allclose(pr.limited_unit(np.array([9.0, -9.0]), np.array([9.0, -9.0]), 2.0),
                       [2 * pr.sigmoid(3.404) * 3, -9 * pr.sigmoid(-9 * 1.702) * -1])
    w = {"router": np.eye(3), "router.b": np.array([0.0, 0.0, 5.0])}
    ids, wts = pr.route(np.array([[1.0, 2.0, 0.0]]), w, "", 2)
    assert ids.tolist() == [[2, 1]] and np.allclose(wts, np.exp([5.0, 2.0]) / np.exp([5.0, 2.0]).sum())


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

    cfg_fault("residual factor", lambda c: c.update(residual_mult=c["residual_mult"] * 1.5))
    cfg_fault("embedding scale", lambda c: c["embedding"].update(scale=c["embedding"]["scale"] * 2))
    cfg_fault("eps", lambda c: c["norm"].update(eps=0.5))
    w_fault("final norm's bias off", "final.norm.b", lambda a: a * 0)
    flip = lambda a: a[:, ::-1].copy()
    for i, layer in enumerate(cfg["layers"]):
        m, kind, p, at = layer["mixer"], layer["type"], f"l{i}.", f"layer {i}: "
        for q in (1, 2) if layer.get("mlp") else (1,):
            w_fault(f"{at}norm {q} without its bias", f"{p}norm{q}.b", lambda a: a * 0)
            w_fault(f"{at}sublayer {q} unscaled", f"{p}ls{q}", lambda a: a * 0 + 1)
            w_fault(f"{at}input convolution {q} off", f"{p}canon{q}", lambda a: a * 0)
            w_fault(f"{at}input convolution {q} turned round", f"{p}canon{q}", flip)
            w_fault(f"{at}a stream not written in {q}", f"{p}hc{q}.out", lambda a: a * (np.arange(len(a)) > 0))
            if cfg["streams"] > 1:
                if i > 0:  # the first layer finds the streams alike, or nearly so: its norms take the factor away
                    w_fault(f"{at}signs of the streams read in {q}", f"{p}hc{q}.in", np.abs)
                w_fault(f"{at}mixing {q} the wrong way round", f"{p}hc{q}.mix", lambda a: a.T.copy())
        if kind == "attention":
            cfg_fault(at + "scale", lambda c, i=i: c["layers"][i]["mixer"].update(scale=m["scale"] * 2))
            cfg_fault(at + "rotary base", lambda c, i=i: c["layers"][i]["mixer"]["rot"].update(base=m["rot"]["base"] * 10))
            cfg_fault(at + "half the rotated numbers", lambda c, i=i: c["layers"][i]["mixer"]["rot"].update(dims=m["rot"]["dims"] // 4 * 2))
            w_fault(at + "sinks far below every score", p + "mix.sink", lambda a: a - 60)
            w_fault(at + "sinks of zero", p + "mix.sink", lambda a: a * 0)
        else:
            w_fault(at + "decays", p + "mix.A_log", lambda a: a + 1.5)
            w_fault(at + "step bias", p + "mix.dt_bias", lambda a: a + 1.0)
            w_fault(at + "state forgotten at once", p + "mix.A_log", lambda a: a * 0 + 9)
            w_fault(at + "gain dropped", p + "mix.norm", lambda a: a * 0 + 1)
        if kind == "delta":
            w_fault(at + "write strength", p + "mix.b", lambda a: a * 0)
            w_fault(at + "gate", p + "mix.g", lambda a: -a)
            for n in ("q", "k", "v"):
                if m["conv"] > 1:
                    w_fault(f"{at}{n}'s convolution turned round", f"{p}mix.{n}.conv", flip)
        if kind == "mamba2":
            w_fault(at + "skip", p + "mix.D", lambda a: a * 0)
            w_fault(at + "convolution's bias", p + "mix.conv.b", lambda a: a * 0)
            w_fault(at + "convolution turned round", p + "mix.conv", flip)
            if m["norm_groups"] > 1:
                cfg_fault(at + "one norm for all parts", lambda c, i=i: c["layers"][i]["mixer"].update(norm_groups=1))
        mlp = layer.get("mlp")
        if mlp and mlp["kind"] == "dense":
            for j in range(4):
                w_fault(f"{at}coefficient {j}", p + "mlp.act", lambda a, j=j: a * (np.arange(4) != j))
        elif mlp:
            cfg_fault(at + "limit", lambda c, i=i: c["layers"][i]["mlp"]["expert"].update(limit=mlp["expert"]["limit"] * 0.4))
            if mlp["router"]["experts"] > 1:
                w_fault(at + "router's bias", p + "mlp.router.b", lambda a: a * 0)
    return out


@pytest.mark.parametrize("case", sorted(rc.CASES))
def test_every_constant_and_tensor_kind_moves_the_logits(case):
    """Every fault moves the logits by more than the GPU tests let a bfloat16 engine differ (tests/test_rudolix_gpu.py: no
    position beyond three times the largest gap that rounding the stored activations opens, at most a fifth of the
    positions beyond three times the gap's 80th percentile)."""
    cfg = rc.CASES[case]
    w = rc.draw_weights(cfg, 26, calm=True)
    toks = random_tokens(5, 150, cfg["vocab"])
    ref = pr.forward(toks, w, cfg)
    gap = np.abs(pr.forward(toks, w, cfg, r=pr.to_bf16) - ref).max(axis=1)
    faults = _faults(cfg)
    assert len(faults) >= 35
    missed = []
    for name, c, change in faults:
        err = np.abs(pr.forward(toks, change(w) if change else w, c) - ref).max(axis=1)
        if "streams read" in name:  # after one update the streams are still nearly proportional: single precision tells
            if not err.max() > 30 * TOL_F32 * np.abs(ref).max():
                missed.append(name)
        elif not (err.max() > 3.0 * gap.max() or int((err > 3.0 * np.percentile(gap, 80)).sum()) > len(toks) // 5):
            missed.append(name)
    assert not missed, f"case {case}: no more than rounding may: {missed}"


@pytest.mark.parametrize("case", sorted(rc.CASES))
def test_what_a_sequence_carries_reaches_far_on(case):
    """The first token shows in the logits a hundred tokens later (a state or a cache that loses its start would not go
    unseen in single precision)."""
    cfg = rc.CASES[case]
    w = rc.draw_weights(cfg, 26)
    toks = random_tokens(6, 140, cfg["vocab"])
    other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    far = np.abs(pr.forward(toks, w, cfg) - pr.forward(other, w, cfg)).max(axis=1)[100:]
    assert far.min() > 1e-4 * np.abs(pr.forward(toks, w, cfg)).max()


# ---- the library's host side ---------------------------------------------------------------------------
def test_the_configuration_becomes_blocks_and_the_designs_tensor_names():
    from bitnet_c_b200.config import architecture_of
    from bitnet_c_b200.engine.model import parameter_table
    for name, cfg in rc.CASES.items():
        arch = architecture_of(cfg)
        assert arch.name == "Rudolix"
        spec = arch.to_spec(arch.read_config(cfg))
        assert len(spec.blocks) == len(spec.schedule) == len(cfg["layers"])
        assert spec.streams == cfg["streams"] and spec.tie_embeddings and spec.embedding_scale == cfg["embedding"]["scale"]
        table = parameter_table(spec)
        names = {arch.tensor_name(p): tuple(s.shape) for p, s in table.items() if not s.optional}
        assert names == {n: tuple(s) for n, s in rc.tensor_shapes(cfg).items()}, name
        assert not any(s.integer for s in table.values())
        # of a sublayer that is left out the file may hold tensors all the same
        spare = {arch.tensor_name(p) for p, s in table.items() if s.optional}
        want = {f"l{i}.{n}" for i, l in enumerate(cfg["layers"]) if l.get("mlp") is None
                for n in ("norm2", "norm2.b", "ls2", "hc2.in", "hc2.out", "hc2.mix", "canon2")}
        assert spare == want


def test_mixers_and_feed_forwards_carry_every_constant_of_the_configuration():
    from bitnet_c_b200.config import architecture_of
    arch = architecture_of(rc.CASE_A)
    spec = arch.to_spec(arch.read_config(rc.CASE_A))
    att, delta, ssm = spec.blocks[0].mixer, spec.blocks[1].mixer, spec.blocks[2].mixer
    assert (att.n_heads, att.n_kv_heads, att.head_dim, att.v_head_dim, att.scale, att.sink) == (6, 2, 16, 24, 0.4, True)
    assert (att.position.dims, att.position.base, att.position.pairing, att.position.factor) == (8, 1000.0, "halves", 1.0)
    assert (delta.n_heads, delta.n_kv_heads, delta.head_dim, delta.v_head_dim, delta.conv_taps, delta.norm_eps) == (6, 3, 12, 20, 3, 1e-5)
    assert (ssm.n_heads, ssm.n_groups, ssm.state, ssm.v_head_dim, ssm.conv_taps, ssm.norm_groups) == (4, 2, 24, 12, 5, 2)
    assert spec.blocks[2].ffn is None and (spec.blocks[1].ffn.kind, spec.blocks[1].ffn.intermediate) == ("poly_mlp", 56)
    moe = spec.blocks[0].ffn
    assert (moe.n_experts, moe.top, moe.expert_ff, moe.expert_limit, moe.slope) == (5, 2, 24, 1.5, 1.702)
    assert moe.router_bias and moe.renormalise and moe.scores == "softmax" and not moe.weight_on_input
    assert all((b.streams, b.residual_mult, b.input_taps, b.mixer_norm.eps) == (3, 0.7, 4, 1e-5) for b in spec.blocks)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(dim=300), "dim"),
    (lambda c: c["layers"][2]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][2]["mixer"].update(groups=3), "multiple"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "kind"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
])
def test_configurations_that_cannot_be_built_are_refused_by_name(change, message):
    from bitnet_c_b200.config import ConfigError, architecture_of
    cfg = copy.deepcopy(rc.CASE_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        architecture_of(cfg).read_config(cfg)


def test_a_run_keeps_several_states_by_name_beside_its_keys_and_values():
    import torch
    from bitnet_c_b200.cache import Cache
    from bitnet_c_b200.config import architecture_of
    from bitnet_c_b200.csrc import ops
    from bitnet_c_b200.engine import Model
    arch = architecture_of(rc.CASE_A)
    model = Model(arch.to_spec(arch.read_config(rc.CASE_A)), dtype="bfloat16", device=None)
    cache = model.new_cache(max_tokens=64 * 8, max_seqs=2, allocate=False)
    want = {(i, f"canon{q}") for i, l in enumerate(rc.CASE_A["layers"]) for q in ((1, 2) if l["mlp"] else (1,))}
    want |= {(i, "mixer") for i, l in enumerate(rc.CASE_A["layers"]) if l["type"] != "attention"}
    assert set(cache.state_requests) == want
    assert cache.state_requests[(0, "canon1")].shape == (3, 64) and cache.state_requests[(0, "canon1")].dtype == torch.bfloat16
    r = cache.state_requests[(1, "mixer")]
    assert r.shape == (ops.gated_state_floats(6, 3, 12, 20, 3),) and r.dtype == torch.float32
    assert len(cache.groups) == 1 and cache.groups[0].request.v_dim == 24
    # tensors by name, zeroed when a slot is opened
    c = Cache([None, None], [None, None], [{"a": r, "b": cache.state_requests[(0, "canon1")]}, r], 128, 128, torch.float32, "cpu")
    for t in c.states.values():
        t.fill_(3.0)
    s = c.open()
    assert set(c.state(0)) == {"a", "b"} and c.state(1).shape[1:] == r.shape
    assert all(float(t[s].float().abs().max()) == 0.0 and float(t[1 - s].float().min()) == 3.0 for t in c.states.values())


def test_random_weights_of_the_design_have_its_tensors_only(tmp_path):
    import bitnet_c_b200 as bn
    from bitnet_c_b200.weights.safetensors_io import SafetensorsFile
    folder = bn.write_random_model(str(tmp_path / "m"), rc.CASE_A, seed=5)
    f = SafetensorsFile(str(tmp_path / "m" / "model.safetensors"))
    try:
        assert {n: tuple(f.entries[n].shape) for n in f.names()} == {n: tuple(s) for n, s in rc.tensor_shapes(rc.CASE_A).items()}
        mix = f.read("l0.hc1.mix").float().numpy()
        assert np.abs(mix - np.eye(3)).max() < 0.6 and not np.array_equal(mix, np.eye(3))
    finally:
        f.close()
    assert json.load(open(tmp_path / "m" / "config.json"))["architecture"] == "Rudolix" and folder

"""The Lakadra design on the GPU against its plain statement (tests/plain_lakadra.py): every kernel it brought or extended
alone, then its mixers, then whole models of small sizes (tests/lakadra_cases.py) through the step function, the cache and
its states, the generation loop and the replay program."""
import copy
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import bitnet_c_b200 as bn
import lakadra_cases as lc
import plain_lakadra as pl
from helpers import (BF16_GAP_FACTOR, TOL_F32, collect_trace_output, compare, random_tokens, replay, steps_to_jsonl,
                     trace_batches, trace_chunks, trace_tail, trace_whole)

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", autouse=True)
def _give_device_memory_back():
    """The models and caches of this module leave the allocator's pool when it is done."""
    yield
    import gc
    gc.collect()
    if torch.cuda.is_available():
        torch.cuda.empty_cache()


ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
bf = pl.to_bf16
f32 = lambda a: np.asarray(a, dtype=np.float32).astype(np.float64)


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).to("cuda", dtype)


def ints(a):
    return torch.tensor(list(a), dtype=torch.int32, device="cuda")


# How three sequences of 150, 4 and 67 tokens are cut into steps.
LENGTHS = [150, 4, 67]
PLANS = {"whole": [[150, 4, 67]],
         "around a piece's edge": [[63, 1, 64], [1, 0, 1], [65, 1, 0], [21, 2, 2]],
         "pairs and single tokens": [[2, 2, 2], [1, 1, 1], [1, 1, 1], [100, 0, 20], [1, 0, 1], [2, 0, 2], [43, 0, 40]]}


def _step_arrays(new, at, slots):
    """What a kernel over states is told of a step: which sequences are in it, and their device arrays."""
    live = [s for s, c in enumerate(new) if c]
    counts = [new[s] for s in live]
    tiles = [(i, r) for i, c in enumerate(counts) for r in range(0, c, 64)]
    return live, dict(tok_seq=ints(np.concatenate([np.full(c, i) for i, c in enumerate(counts)])),
                      seq_start=ints(np.concatenate([[0], np.cumsum(counts)])), seq_pos0=ints([at[s] for s in live]),
                      slots=ints([slots[s] for s in live]), n_seqs=len(live), one_token=max(counts) == 1,
                      tile_seq=ints(i for i, _ in tiles), tile_row0=ints(r for _, r in tiles))


# ---- kernels alone -----------------------------------------------------------------------------------
@pytest.mark.parametrize("blocks,part,taps", [(1, 8, 4), (3, 5, 2), (4, 16, 1), (2, 130, 16), (16, 128, 4), (1, 300, 3), (40, 72, 2)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_gated_recurrence_however_the_tokens_are_cut(cuda_device, blocks, part, taps, dtype):
    """Unequal sequences in scattered slots, in runs that end before, on and behind the edge of a piece, in pairs, and one
    token at a time; the result goes, with a factor, into columns of a wider matrix whose other columns stay; slots that are
    in no step keep what they hold."""
    from bitnet_c_b200.csrc import ops
    n, t = blocks * part, DT[dtype]
    rng = np.random.default_rng(n * 100 + taps)
    conv, conv_b, lam = f32(0.6 * rng.standard_normal((n, taps))), f32(0.3 * rng.standard_normal(n)), f32(rng.uniform(-7, 0, n))
    ra, ri = (bf(1.5 * rng.standard_normal((blocks, part, part)) / np.sqrt(part)) for _ in range(2))
    rb, ib = (f32(rng.standard_normal((blocks, part))) for _ in range(2))
    round_ = bf if dtype == "bfloat16" else lambda a: a
    xs, ys = ([bf(rng.standard_normal((m, n))) for m in LENGTHS] for _ in range(2))
    want = []
    for x, y in zip(xs, ys):
        u = round_(pl.causal_convolution(x, conv, conv_b))
        want.append(1.3 * pl.gelu_tanh(y) * pl.gated_linear_states(u, ra, rb, ri, ib, lam))
    scale = max(np.abs(a).max() for a in want)
    w_gates, gate_b = dev(np.concatenate([ra, ri], axis=1), t), dev(np.concatenate([rb, ib], axis=1))
    slots = [3, 0, 4]
    for what, steps in PLANS.items():
        state = torch.zeros((6, ops.gated_linear_floats(n, taps)), dtype=torch.float32, device="cuda")
        state[1].fill_(7.0)
        at = [0, 0, 0]
        for new in steps:
            live, step = _step_arrays(new, at, slots)
            cat = lambda zs: np.concatenate([zs[s][at[s]:at[s] + new[s]] for s in live])
            T = sum(new)
            rows = dev(np.concatenate([np.full((T, 3), 1e3), cat(ys), cat(xs)], axis=1), t)
            out = torch.full((T, n + 9), 5.0, dtype=t, device="cuda")
            ops.gated_linear(rows[:, 3 + n:], rows[:, 3: 3 + n], dev(conv.T.copy()), dev(conv_b), w_gates, gate_b, dev(lam), state,
                             out=out[:, 2: 2 + n + 4], scale=1.3, tail=4, **step)
            got = out.float().cpu().numpy()
            assert (got[:, :2] == 5.0).all() and (got[:, n + 6:] == 5.0).all() and (got[:, n + 2: n + 6] == [1, 1, 0, 0]).all()
            ref = np.concatenate([want[s][at[s]:at[s] + new[s]] for s in live])
            err = np.abs(got[:, 2: 2 + n] - ref)
            tol = 1e-4 if dtype == "float32" else 2.0 ** -8
            # in bfloat16 a number of u that falls on the border between two may be rounded the other way: a few may be off by more
            assert np.isfinite(got).all() and np.percentile(err, 99.5) < tol * max(1.0, scale) and err.max() < (tol if dtype == "float32" else 0.02) * max(1.0, scale), \
                f"{what}, step {new}: {err.max():.3e} of {scale:.2f}"
            for s in live:
                at[s] += new[s]
        assert at == LENGTHS and bool((state[1] == 7.0).all()) and bool((state[2] == 0.0).all())


@pytest.mark.parametrize("blocks,part", [(3, 24), (60, 48), (2, 288)])
def test_the_gated_recurrence_of_many_sequences_at_once(cuda_device, blocks, part):
    """Nineteen sequences of unequal lengths, then one token each, three times."""
    from bitnet_c_b200.csrc import ops
    n, taps, S = blocks * part, 4, 19
    rng = np.random.default_rng(n)
    conv, conv_b, lam = f32(0.6 * rng.standard_normal((n, taps))), f32(0.3 * rng.standard_normal(n)), f32(rng.uniform(-7, 0, n))
    ra, ri = (bf(1.5 * rng.standard_normal((blocks, part, part)) / np.sqrt(part)) for _ in range(2))
    rb, ib = (f32(rng.standard_normal((blocks, part))) for _ in range(2))
    lens = [1 + 5 * (s % 4) for s in range(S)]
    xs, ys = ([bf(rng.standard_normal((m + 3, n))) for m in lens] for _ in range(2))
    want = [pl.gelu_tanh(y) * pl.gated_linear_states(pl.causal_convolution(x, conv, conv_b), ra, rb, ri, ib, lam) for x, y in zip(xs, ys)]
    scale = max(np.abs(a).max() for a in want)
    state = torch.zeros((S, ops.gated_linear_floats(n, taps)), dtype=torch.float32, device="cuda")
    at, slots = [0] * S, rng.permutation(S).tolist()
    for new in (lens, [1] * S, [1] * S, [1] * S):
        live, step = _step_arrays(new, at, slots)
        cat = lambda zs: dev(np.concatenate([zs[s][at[s]:at[s] + new[s]] for s in live]))
        out = torch.empty((sum(new), n), device="cuda")
        ops.gated_linear(cat(xs), cat(ys), dev(conv.T.copy()), dev(conv_b), dev(np.concatenate([ra, ri], axis=1)), dev(np.concatenate([rb, ib], axis=1)),
                         dev(lam), state, out=out, **step)
        ref = np.concatenate([want[s][at[s]:at[s] + new[s]] for s in live])
        assert np.abs(out.cpu().numpy() - ref).max() < 1e-4 * max(1.0, scale)
        at = [a + c for a, c in zip(at, new)]


def _lightning_inputs(rng, H, d, dv):
    z = lambda m: {"q": bf(rng.standard_normal((m, H * d))), "k": bf(rng.standard_normal((m, H * d))), "v": bf(rng.standard_normal((m, H * dv)))}
    return [z(m) for m in LENGTHS]


def _run_lightning(zs, H, d, dv, decay, steps, dtype, chunks, slots=(3, 0, 4), state=None):
    from bitnet_c_b200.csrc import ops
    at, got = [0] * len(zs), [np.zeros((z["q"].shape[0], H * dv)) for z in zs]
    logs = dev(np.log(np.maximum(decay, 1e-40)))
    if state is None:
        state = torch.zeros((6, ops.gated_state_floats(H, H, d, dv, 1)), dtype=torch.float32, device="cuda")
    for new in steps:
        live, step = _step_arrays(new, at, slots)
        if not chunks:
            step.update(tile_seq=None, tile_row0=None)
        rows = dev(np.concatenate([np.concatenate([zs[s][k][at[s]:at[s] + new[s]] for k in ("v", "k", "q")], axis=1) for s in live]), DT[dtype])
        o = ops.gated_state(rows, H * (dv + d), H * dv, 0, None, 0, -1, None, None, None, None, None, state, heads=H, groups=H, dim=d, vdim=dv,
                            log_decay=logs, **step).cpu().numpy()
        r = 0
        for s in live:
            got[s][at[s]:at[s] + new[s]] = o[r:r + new[s]]
            r += new[s]
            at[s] += new[s]
    assert at == [len(g) for g in got]
    return got, state


@pytest.mark.parametrize("H,d,dv", [(4, 16, 24), (1, 40, 136), (3, 10, 7), (2, 132, 40), (2, 256, 8), (5, 64, 64), (8, 128, 128)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_states_under_fixed_decays_however_the_tokens_are_cut(cuda_device, H, d, dv, dtype):
    """Token by token and piece by piece; decays from none (everything is kept) to all (only the token itself counts)."""
    rng = np.random.default_rng(H * 1000 + d)
    zs = _lightning_inputs(rng, H, d, dv)
    decay = np.array([0.0, 1.0, 0.999, 0.6, 0.97, 0.9, 0.99, 0.3])[:H] if H > 1 else np.array([0.98])
    want = []
    for z in zs:
        q, k, v = (pl.silu(z[n]).reshape(len(z[n]), H, -1) for n in "qkv")
        want.append(np.stack([pl.lightning_state(q[:, h], k[:, h], v[:, h], decay[h]) for h in range(H)], axis=1).reshape(len(q), -1))
    scale = max(np.abs(a).max() for a in want)
    for what, steps in PLANS.items():
        for chunks in (False, True):
            if chunks and d % 4:
                continue
            got, state = _run_lightning(zs, H, d, dv, decay, steps, dtype, chunks)
            for s, (a, b) in enumerate(zip(got, want)):
                err = np.abs(a - b).max(axis=1)
                assert np.isfinite(a).all() and err.max() < 1e-4 * max(1.0, scale), f"{what}, pieces {chunks}: sequence {s}, token {int(err.argmax())}: {err.max():.3e} of {scale:.2f}"
            assert bool((state[1] == 0.0).all()) and bool((state[2] == 0.0).all())


def test_one_write_among_hundreds_of_tokens_is_kept_or_forgotten_by_its_decay(cuda_device):
    """All values are zero but one token's, planted at the start and at both sides of pieces' edges: the head with a slow
    decay reads it back at the end, the fast one has forgotten it, in prompts and in decoding."""
    H, d, dv, T = 2, 32, 32, 300
    rng = np.random.default_rng(3)
    for at in (0, 1, 63, 64, 65, 128, 191, 255, 256):
        z = {k: bf(rng.standard_normal((T, H * n))) for k, n in (("q", d), ("k", d), ("v", dv))}
        z["v"][:] = 0.0
        z["v"][at] = bf(rng.standard_normal(H * dv) + 4.0)
        z["q"][-1] = z["k"][at] = bf(np.abs(z["k"][at]) + 1.0)
        decay = np.array([0.999, 0.5])
        q, k, v = (pl.silu(z[n]).reshape(T, H, -1) for n in "qkv")
        want = np.stack([pl.lightning_state(q[:, h], k[:, h], v[:, h], decay[h]) for h in range(H)], axis=1)
        assert np.abs(want[-1, 0]).min() > 10 and (at > 250 or np.abs(want[-1, 1]).max() < 1e-8)
        for steps in ([[T]], [[at + 1], [T - 1 - at]] if at < T - 1 else [[T]], [[290]] + [[1]] * 10):
            (got,), _ = _run_lightning([z], H, d, dv, decay, steps, "bfloat16", True, slots=(2,))
            err = np.abs(got - want.reshape(T, -1)).max()
            assert err < 2e-4 * np.abs(want).max(), f"planted at {at}, steps {steps[:2]}: {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("length", [7, 66, 200, 1030, 4096])
def test_one_norm_over_all_heads_and_a_logistic_gate(cuda_device, dtype, length):
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(length)
    o, z, gain = f32(5 * rng.standard_normal((33, length))), bf(2 * rng.standard_normal((33, length))), f32(1 + 0.3 * rng.standard_normal(length))
    pad = -length % 8
    rows = dev(np.concatenate([np.zeros((33, 8)), z, np.zeros((33, pad))], axis=1), DT[dtype])
    got = ops.state_output(dev(o), rows[:, 8: 8 + length], dev(gain), 1, 1e-5, False, DT[dtype], logistic=True).float().cpu().numpy()
    want = pl.unit_rms(o, 1e-5) * gain * pl.sigmoid(z)
    assert np.abs(got - want).max() < (2e-5 if dtype == "float32" else 2.0 ** -7) * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,groups,keep,top", [(6, 3, 2, 2), (18, 3, 2, 3), (8, 8, 3, 3), (40, 4, 1, 10), (5, 1, 1, 5), (1, 1, 1, 1), (320, 80, 7, 8), (1024, 2, 2, 32)])
def test_the_router_chooses_by_corrected_scores_within_groups(cuda_device, dtype, experts, groups, keep, top):
    """Corrections of both signs and all negative; without them; the weights are the uncorrected scores; a last row of the
    router's matrix gives a gate."""
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(experts + top)
    W, T, t = 72, 150, DT[dtype]
    h, w = bf(rng.standard_normal((T, W))), bf(rng.standard_normal((experts + 1, W)) / 8)
    z = h @ w.T
    for shift, spread in ((0.0, 0.3), (-1.5, 0.3), (0.0, 0.0)):
        c = f32(shift + spread * rng.standard_normal(experts))
        ids, weights, gate = ops.moe_route(dev(h, t), dev(w, t), top, softmax=True, correction=dev(c), groups=groups, keep=keep, gate=True)
        want_ids, want_w = pl.choose_experts(z[:, :experts], c, top, groups, keep)
        e = np.exp(z[:, :experts] - z[:, :experts].max(1, keepdims=True))
        s = e / e.sum(1, keepdims=True)
        got = ids.cpu().numpy()
        # where two choices are as good as equal rounding decides: the chosen scores must be those of the plain choice
        per = np.take_along_axis(s + c, got, 1)
        ref = np.take_along_axis(s + c, want_ids, 1)
        assert np.abs(per - ref).max() < 1e-5
        same = got == want_ids
        assert same.mean() > 0.98 and np.abs(weights.cpu().numpy() - want_w)[same].max() < 2e-5
        assert np.abs(weights.cpu().numpy() - np.take_along_axis(s, got, 1)).max() < 2e-5
        assert all(len(set(r)) == top for r in got.tolist())
        assert np.abs(gate.cpu().numpy() - pl.sigmoid(z[:, experts])).max() < 2e-5
        # the same behind a product of its own
        logits = torch.cat([dev(z), torch.full((T, 7), float("nan"), device="cuda")], dim=1)
        again = ops.moe_choose(logits, experts, top, softmax=True, correction=dev(c), groups=groups, keep=keep, gate=True)
        assert (again[0].cpu().numpy() == want_ids).mean() > 0.98 and np.abs(again[1].cpu().numpy() - np.take_along_axis(s, again[0].cpu().numpy(), 1)).max() < 2e-5
        assert np.abs(again[2].cpu().numpy() - pl.sigmoid(z[:, experts])).max() < 2e-5
    plain = ops.moe_route(dev(h, t), dev(w[:experts], t), top, softmax=True)
    assert len(plain) == 2 and (plain[0].cpu().numpy() == np.argsort(-z[:, :experts], axis=1, kind="stable")[:, :top]).mean() > 0.98


def test_a_router_of_a_wide_model(cuda_device):
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(1)
    h, w, c = bf(rng.standard_normal((5, 12000))), bf(rng.standard_normal((9, 12000)) / 100), f32(0.1 * rng.standard_normal(8))
    ids, weights, gate = ops.moe_route(dev(h, torch.bfloat16), dev(w, torch.bfloat16), 3, softmax=True, correction=dev(c), groups=4, keep=2, gate=True)
    want_ids, want_w = pl.choose_experts((h @ w.T)[:, :8], c, 3, 4, 2)
    assert (ids.cpu().numpy() == want_ids).all() and np.abs(weights.cpu().numpy() - want_w).max() < 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,experts,identity,top,ff,shared", [(64, 5, 1, 2, 24, 40), (50, 3, 3, 3, 13, 7), (96, 4, 0, 4, 32, 0), (128, 9, 7, 1, 48, 16), (40, 1, 4, 2, 8, 8)])
def test_experts_without_a_gate_identity_experts_and_a_gated_shared_one(cuda_device, dtype, W, experts, identity, top, ff, shared):
    """Few rows (streamed) and many (sorted, in equal blocks or packed), evenly used or nearly all on one expert, and all on
    identity experts."""
    from bitnet_c_b200.config import MoeSpec
    from bitnet_c_b200.engine.batch import SeqStep, pack_step
    from bitnet_c_b200.parts import BuildContext, build_part
    t = DT[dtype]
    rng = np.random.default_rng(W + experts)
    mlp = lc.moe(experts, identity, top, 1, 1, ff, shared)
    if not shared:
        mlp["shared"] = None
    cfg = {"width": W, "vocab": 8, "layers": [{"type": "lightning", "mixer": {"heads": 1, "dim": 4, "vdim": 4, "decay": [0.5]}, "mlp": mlp}]}
    w = {n[7:]: a for n, a in lc.draw_weights(cfg, 5, calm=True).items() if n.startswith("l0.mlp.")}
    spec = MoeSpec(width=W, n_experts=experts, top=top, expert_ff=ff, expert_limit=0.0, shared_ff=shared, weight_on_input=False, scores="softmax",
                   activation="relu2", correction=True, identity=identity, shared_gate=shared > 0)
    ffn = build_part("ffn", spec, BuildContext(dtype=t, device=torch.device("cuda:0")))
    n_out = experts + identity
    kinds = {"as drawn": w["correction"], "one expert before all": np.where(np.arange(n_out) == 0, 5.0, w["correction"]),
             "identity experts before all": np.where(np.arange(n_out) >= experts, 50.0 + np.arange(n_out), w["correction"])}
    for kind, corr in kinds.items():
        ffn.bind({n: dev(corr if n == "correction" else a, t) for n, a in w.items()})
        wk = {**w, "correction": bf(corr)}
        for T, grouped in ((1, True), (3, True), (40, True), (300, True), (40, False), (300, False)):
            ffn.USE_GROUPED = grouped
            h = bf(rng.standard_normal((T, W)))
            ctx = pack_step([SeqStep(0, [0] * T)], [0], torch.device("cuda:0"))
            got = ffn.forward(dev(h, t), ctx).cpu().numpy()
            want = pl.experts(h, wk, "", mlp)
            tol = 2e-5 if dtype == "float32" else 0.02
            assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), f"{kind}, {T} tokens"


@pytest.mark.parametrize("M", [1, 7, 16, 17, 40, 64, 65, 300, 1100])
@pytest.mark.parametrize("N,K", [(24, 64), (300, 256), (1040, 512), (129, 50)])
def test_products_with_a_bias_and_with_squared_relu(cuda_device, M, N, K):
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(M * 1000 + N)
    x, w, b = bf(rng.standard_normal((M, K))), bf(rng.standard_normal((N, K)) / np.sqrt(K)), bf(3 * rng.standard_normal(N))
    want = x @ w.T + b
    for dtype in ("float32", "bfloat16"):
        t = DT[dtype]
        for tc in (True, False):
            ops.USE_TCGEN05, before = tc, ops.USE_TCGEN05
            try:
                for out_dtype in {t, torch.float32}:
                    tol = 2e-5 if out_dtype == torch.float32 else 2.0 ** (-8 if K % 8 == 0 else -7)  # (odd sizes: the library's choice)
                    got = ops.linear(dev(x, t), dev(w, t), out_dtype=out_dtype, bias=dev(b)).float().cpu().numpy()
                    assert np.abs(got - want).max() < tol * np.abs(want).max() * 1.1, (dtype, tc, out_dtype)
                got = ops.linear(dev(x, t), dev(w, t), act=ops.ACT_RELU2).float().cpu().numpy()
                ref = np.square(np.maximum(x @ w.T, 0))
                assert np.abs(got - ref).max() < (2e-5 if dtype == "float32" else 2.0 ** -6) * np.abs(ref).max(), (dtype, tc)
            finally:
                ops.USE_TCGEN05 = before
    ops.check_tc_status(torch.device("cuda:0"))


@pytest.mark.parametrize("counts", [[300, 0, 5, 256, 1, 0], [0, 0, 0], [1], [257, 255, 513], [0, 700], [3] * 40, [0] * 1023 + [9]])
@pytest.mark.parametrize("N,K", [(8, 64), (264, 72), (512, 256), (1000, 40)])
def test_products_of_groups_of_rows_each_with_its_own_matrix(cuda_device, counts, N, K):
    """Groups of none, one and many rows, around a tile's edge; rows behind the last group are left alone whatever lies there."""
    from bitnet_c_b200.csrc import ops
    if len(counts) * N * K > 4e7:
        pytest.skip("a large stack of matrices adds nothing here")
    g = torch.Generator(device="cuda").manual_seed(sum(counts) + N)
    rows = sum(counts) + 300
    x = torch.randn((rows, K), device="cuda", generator=g).bfloat16()
    x[sum(counts):] = float("nan")
    w = (torch.randn((len(counts), N, K), device="cuda", generator=g) / K ** 0.5).bfloat16()
    offsets = ints(np.concatenate([[0], np.cumsum(counts)]))
    for act in (0, ops.ACT_RELU2):
        got = ops.grouped_product(x, w, offsets, act=act)
        at = 0
        for e, c in enumerate(counts):
            ref = x[at:at + c].float() @ w[e].float().T
            ref = torch.relu(ref) ** 2 if act else ref
            if c:
                assert bool(torch.isfinite(got[at:at + c]).all()) and float((got[at:at + c].float() - ref).abs().max()) < 2.0 ** -7 * float(ref.abs().max()), f"group {e}"
            at += c
    ops.check_tc_status(torch.device("cuda:0"))


@pytest.mark.parametrize("H,G,d,dv,window", [(4, 2, 160, 128, 0), (3, 3, 192, 128, 0), (2, 2, 144, 64, 0), (4, 1, 176, 48, 100), (8, 8, 192, 96, 64), (4, 2, 64, 64, 70), (2, 1, 128, 128, 1)])
def test_wide_keys_gates_and_columns_of_a_wider_matrix_on_tcgen05(cuda_device, H, G, d, dv, window):
    """Keys of up to 192 numbers, a gate per head, a factor, a score of zero in the denominator; the result goes into columns of
    a wider matrix; pieces behind cached tokens, unequal runs; against the general kernel in float32."""
    from bitnet_c_b200.csrc import ops
    lens, new = [300, 131, 40, 1], [300, 70, 17, 1]
    g = torch.Generator(device="cuda").manual_seed(d + dv)
    n, pages = sum(new), [(m + 63) // 64 for m in lens]
    q = torch.randn((n, H * d + H + 8 - H % 8), device="cuda", generator=g).bfloat16() * 2
    kc, vc = (torch.randn((sum(pages) + 1, G, 64, w), device="cuda", generator=g).bfloat16() for w in (d, dv))
    table, at = torch.zeros((4, max(pages)), dtype=torch.int32, device="cuda"), 1
    for i, p in enumerate(pages):
        table[i, :p] = torch.arange(at, at + p, device="cuda")
        at += p
        vc[table[i, p - 1].long(), :, (lens[i] - 1) % 64 + 1:] = float("nan")  # behind the sequence's last position
    start = ints(np.concatenate([[0], np.cumsum(new)]))
    pos0, slots = ints(a - b for a, b in zip(lens, new)), ints(range(4))
    tok_seq = ints(np.concatenate([np.full(c, i) for i, c in enumerate(new)]))
    tok_pos = ints(np.concatenate([np.arange(m - c, m) for m, c in zip(lens, new)]))
    tiles = [(i, r) for i, c in enumerate(new) for r in range(0, c, 128)]
    sink, gate = torch.zeros(H, device="cuda"), q[:, H * d:]
    wide = torch.full((n, H * dv + 24), 5.0, dtype=torch.bfloat16, device="cuda")
    ops.attention_prefill_tc(q, q.shape[1], wide[:, 8:], H, G, d, d ** -0.5, window, ints(i for i, _ in tiles), ints(r for _, r in tiles), start, pos0,
                             slots, table, kc, vc, precise=True, sink=sink, gate=gate, gate_stride=q.shape[1], out_scale=0.7)
    ref = torch.empty((n, H * dv), dtype=torch.float32, device="cuda")
    qf = q.float().contiguous()
    ops.attention_general(qf, q.shape[1], ref, n, H, G, d, d ** -0.5, window, tok_seq, tok_pos, slots, table, kc.float(), vc.float(), sink=sink,
                          gate=qf[:, H * d:], gate_stride=q.shape[1], out_scale=0.7)
    got = wide.float()
    assert bool((got[:, :8] == 5.0).all()) and bool((got[:, 8 + H * dv:] == 5.0).all())
    err = (got[:, 8: 8 + H * dv] - ref).abs()
    assert bool(torch.isfinite(got).all()) and bool((err <= 2.0 ** -8 * ref.abs() + 2e-4).all()), float(err.max())
    ops.check_tc_status(torch.device("cuda:0"))


# ---- mixers alone --------------------------------------------------------------------------------------
def _run_mixers(mixers, cache_of, hs, plans, t, check):
    """Mixers as the entries of a schedule over one cache poisoned with NaN and Inf, each fed the same rows: ``check(entry,
    sequence, first position, rows)`` gets every step's results.  ``plans``: lists of steps (new tokens per sequence)."""
    from bitnet_c_b200.cache import Cache
    from bitnet_c_b200.engine.batch import SeqStep, pack_step
    gpu = torch.device("cuda:0")
    cache = Cache([m.cache_request() for m in mixers], cache_of, [m.state_request() for m in mixers], 64 * 24, 4096, t, gpu, max_seqs=len(hs) + 1)
    for g in cache.groups:
        g.k.fill_(float("nan"))
        if g.v is not None:
            g.v.fill_(float("inf"))
    for s in cache.states.values():
        s.fill_(float("nan"))
    for steps in plans:
        slots, at = [cache.open() for _ in hs], [0] * len(hs)
        for new in steps:
            live = [s for s in range(len(hs)) if new[s]]
            for s in live:
                cache.reserve(slots[s], new[s])
            cache.sync()
            ctx = pack_step([SeqStep(slots[s], [0] * new[s]) for s in live], [at[s] for s in live], gpu)
            rows = dev(np.concatenate([hs[s][at[s]:at[s] + new[s]] for s in live]), t)
            for e, m in enumerate(mixers):
                got, r = m.forward(rows, ctx, cache.view(e), cache.state(e)).float().cpu().numpy(), 0
                for s in live:
                    check(e, s, at[s], got[r:r + new[s]])
                    r += new[s]
            for s in live:
                cache.advance(slots[s], new[s])
                at[s] += new[s]
        for s in slots:
            cache.close(s)


def _bound(spec, w, t):
    from bitnet_c_b200.parts import BuildContext, build_part

    def bind(part, prefix=""):
        names = [n for n in part.params()]
        if names:
            part.bind({n: dev(w[prefix + n], t) for n in names})
        for name, child in part.children().items():
            bind(child, prefix + name + ".")
        part.bound()
    part = build_part("mixer", spec, BuildContext(dtype=t, device=torch.device("cuda:0")))
    bind(part)
    return part


def _spec_of(layer, W, layers=None, i=0):
    from bitnet_c_b200.config import architecture_of
    cfg = {"architecture": "Lakadra", "vocab": 8, "width": W, "norm": {"eps": 1e-5}, "logit_scale": 1.0,
           "layers": layers or [layer]}
    arch = architecture_of(cfg)
    return arch.to_spec(arch.read_config(cfg)).blocks[i].mixer


def _mixer_weights(layers, W, i, seed):
    cfg = {"vocab": 8, "width": W, "layers": layers}
    p = f"l{i}.mix."
    return {n[len(p):]: a for n, a in lc.draw_weights(cfg, seed, calm=True).items() if n.startswith(p)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,dim,vdim,window,dims", [(4, 2, 32, 16, 70, 8), (8, 1, 64, 64, 64, 64), (3, 3, 10, 7, 65, 10), (6, 2, 48, 80, 129, 32),
                                                           (4, 4, 144, 32, 100, 16), (2, 1, 128, 128, 63, 128)])
def test_a_key_at_the_edge_of_the_window(cuda_device, dtype, heads, kv, dim, vdim, window, dims):
    """Keys answer queries, and one token far above the others in size asks for one like itself: ``window`` - 1 tokens back it is
    found, ``window`` tokens back it is not; at several places of pages, in prompts, behind cached tokens and decoded,
    beside other sequences.  The recurrence beside the attention runs along."""
    t, W = DT[dtype], 64
    layer = {"type": "parallel", "mixer": lc.pair(heads, kv, dim, vdim, window, dims, 1e7, 2.0, dim ** -0.5, 40, 4, 3)}
    w = _mixer_weights([layer], W, 0, seed=dim)
    # keys come from the second 21 numbers of a row, values from what follows, queries, alike to keys, from the first 21
    w["left.k"][:, :21] = w["left.k"][:, 42:] = 0.0
    w["left.v"][:, :42] = 0.0
    w["left.q"] = np.repeat(np.roll(w["left.k"], -21, axis=1).reshape(kv, dim, W), heads // kv, axis=0).reshape(heads * dim, W)
    w["left.q.b"], w["left.k.b"] = w["left.q.b"] * 0.1, w["left.k.b"] * 0.1
    w["left.q.b"], w["left.k.b"] = bf(w["left.q.b"]), bf(w["left.k.b"])
    w["right.o"] = bf(w["right.o"] * 0.25)
    left = {n[5:]: a for n, a in w.items() if n.startswith("left.")}
    mixer = _bound(_spec_of(layer, W), w, t)
    assert mixer.together
    rng = np.random.default_rng(dims * dim)
    for far, back in ((0, window - 1), (0, window), (63, window - 1), (64, window), (37, window - 1), (130, window)):
        n = far + back + 1
        hs = [bf(rng.standard_normal((m, W))) for m in (n, 70, 5)]
        other = copy.deepcopy(layer["mixer"]["left"])
        other["mask"]["size"] = window + (1 if back == window else -1)
        for _ in range(60):  # rows whose rotation leaves the score standing out
            hs[0][n - 1][:21] = hs[0][far][21:42] = bf(4.0 * rng.standard_normal(21))
            a, b = (pl.windowed_attention(hs[0], left, "", m)[-1] for m in (layer["mixer"]["left"], other))
            if np.abs(a - b).max() > 0.3 * np.abs(a).max():
                break
        want = [pl.side_by_side(h, w, "", layer["mixer"]) for h in hs]
        assert 0.8 * np.abs(a - b).max() > 0.07 * np.abs(want[0][-1]).max()

        def check(e, s, at, got):
            ref = want[s][at: at + len(got)]
            err = np.abs(got - ref).max(axis=1)
            assert np.isfinite(got).all() and err.max() < (3e-5 if dtype == "float32" else 0.03) * max(1.0, np.abs(ref).max()), \
                f"far {far}, back {back}: sequence {s}, position {at + int(err.argmax())}: {err.max():.3e}"
        last = n - 64 if n > 64 else 1
        _run_mixers([mixer], [None], hs, ([[n, 70, 5]], [[n - 1, 69, 3], [1, 1, 1]], [[last, 64, 2], [n - last - 3, 1, 0], [1, 2, 1], [1, 1, 1], [1, 2, 1]]), t, check)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(4, 16, 16, 16, 48), (3, 9, 6, 7, 19), (4, 64, 32, 64, 256), (2, 128, 64, 128, 192), (8, 32, 32, 80, 96), (2, 48, 16, 32, 320)])
def test_latent_rows_are_found_far_away_by_their_own_layer_and_by_readers(cuda_device, dtype, heads, dim, rot, vdim, rank):
    """Two mixers on one plane of latents, the second without a latent of its own; one key far back stands out, in prompts,
    pieces and decoding."""
    t, W = DT[dtype], 64
    a = lc.latent(heads, dim, rot, vdim, 40, rank, 1.5 * (dim + rot) ** -0.5, 1e6)
    b = lc.latent(heads + 1, dim, rot, vdim, 24, rank, (dim + rot) ** -0.5, 1e6, kv_from=0)
    layers = [{"type": "latent_attention", "mixer": m} for m in (a, b)]
    ws = [_mixer_weights(layers, W, i, seed=rank + i) for i in (0, 1)]
    mixers = [_bound(_spec_of(None, W, layers, i), ws[i], t) for i in (0, 1)]
    assert mixers[0].spec.own_kv and not mixers[1].spec.own_kv
    rng = np.random.default_rng(rank)
    for far in (0, 63, 64, 130):
        hs = [bf(rng.standard_normal((m, W))) for m in (300, 70, 5)]
        # the far row is the one among many whose score under the last query of head 0 is largest
        best, best_gap = hs[0][far], -1.0
        for _ in range(40):
            trial = bf(rng.standard_normal(W) * 3)
            hs[0][far] = trial
            c, kr = pl.latent_rows(hs[0], ws[0], "", a, 1e-5)
            cq = pl.unit_rms(hs[0] @ ws[0]["dq"].T, 1e-5) * ws[0]["dq.norm"]
            q = (cq @ ws[0]["uq"].T).reshape(300, heads, dim + rot)
            s = (c @ ws[0]["uk"].T).reshape(300, heads, dim)[:, 0] @ q[-1, 0, :dim] + kr @ pl.turned(q[..., dim:], 1e6, rot, "neighbours")[-1, 0]
            gap = s[far] - np.delete(s, far).max()
            if gap > best_gap:
                best, best_gap = trial, gap
        hs[0][far] = best
        rows = [pl.latent_rows(h, ws[0], "", a, 1e-5) for h in hs]
        want = [[pl.latent_attention(h, ws[e], "", m, 1e-5, r) for h, r in zip(hs, rows)] for e, m in enumerate((a, b))]

        def check(e, s, at, got):
            ref = want[e][s][at: at + len(got)]
            err = np.abs(got - ref).max(axis=1)
            assert np.isfinite(got).all() and err.max() < (3e-5 if dtype == "float32" else 0.03) * max(1.0, np.abs(ref).max()), \
                f"far {far}, mixer {e}: sequence {s}, position {at + int(err.argmax())}: {err.max():.3e}"
        _run_mixers(mixers, [None, 0], hs, ([[300, 70, 5]], [[64, 69, 3], [66, 1, 1], [170, 0, 1]], [[290, 60, 1]] + [[1, 1, 1]] * 4 + [[6, 6, 0]]), t, check)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixers_of_a_pair_run_alone_too(cuda_device, dtype):
    """The recurrent block and the attention with biases as mixers of their own; and a pair whose left does not share its
    products (lightning attention) runs its two one after the other."""
    from bitnet_c_b200.config import PairSpec
    t, W = DT[dtype], 48
    layers = [{"type": "parallel", "mixer": lc.pair(4, 2, 16, 24, 50, 16, 1e4, 2.0, 0.4, 60, 3, 4)},
              {"type": "lightning", "mixer": {"heads": 3, "dim": 16, "vdim": 8, "decay": [0.5, 0.9, 0.99]}}]
    w = [_mixer_weights(layers, W, i, 9) for i in (0, 1)]
    both = _spec_of(None, W, layers, 0)
    side = lambda name: {n[len(name) + 1:]: a for n, a in w[0].items() if n.startswith(name + ".")}
    m = layers[0]["mixer"]
    rng = np.random.default_rng(4)
    hs = [bf(rng.standard_normal((n, W))) for n in LENGTHS]
    light = lambda h: pl.lightning(h, w[1], "", layers[1]["mixer"], 1e-5)
    cases = [(_bound(both.left, side("left"), t), lambda h: pl.windowed_attention(h, side("left"), "", m["left"])),
             (_bound(both.right, side("right"), t), lambda h: pl.recurrent_block(h, side("right"), "", m["right"])),
             (_bound(PairSpec(left=_spec_of(None, W, layers, 1), right=both.right, left_scale=2.0, right_scale=-1.0),
                     {**{"left." + n: a for n, a in w[1].items()}, **{"right." + n: a for n, a in side("right").items()}}, t),
              lambda h: 2.0 * light(h) - pl.recurrent_block(h, side("right"), "", m["right"]))]
    for mixer, plain in cases:
        want = [plain(h) for h in hs]

        def check(e, s, at, got):
            ref = want[s][at: at + len(got)]
            assert np.isfinite(got).all() and np.abs(got - ref).max() < (3e-5 if dtype == "float32" else 0.03) * max(1.0, np.abs(want[s]).max())
        _run_mixers([mixer], [None], hs, PLANS.values(), t, check)


# ---- whole models --------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """Per case and number format: (folder, weights).  bfloat16 models have routers whose choices rounding leaves alone."""
    out = {}
    for name, cfg in lc.CASES.items():
        for dtype, calm in (("float32", False), ("bfloat16", True)):
            w = lc.draw_weights(cfg, seed=26, calm=calm)
            out[name, dtype] = (lc.write_folder(str(tmp_path_factory.mktemp("lakadra") / (name + dtype)), cfg, w), w)
    return out


_ROUNDED = {}


def _plain_rounded(cfg, w, tokens):
    key = (json.dumps(cfg, sort_keys=True), id(w), tuple(tokens))
    if key not in _ROUNDED:
        _ROUNDED[key] = pl.forward(tokens, w, cfg, r=pl.to_bf16)
    return _ROUNDED[key]


def _check(got, cfg, w, reqs, plain, dtype, what):
    """float32: every position within 1e-4 of the plain logits (relative to the largest).  bfloat16: the bound of a
    request is three times what rounding the stored activations does to the plain statement, taken at the request's
    80th percentile of positions; at most a fifth of a request's positions may lie beyond it, none beyond three
    times the largest gap."""
    for r, per_pos in got.items():
        assert all(np.isfinite(row).all() for row in per_pos.values()), f"{what}: request {r}"
    if dtype == "float32":
        return compare(got, plain, lambda ref: TOL_F32 * max(1.0, float(np.abs(ref).max())), what)
    for r, per_pos in got.items():
        gap = np.abs(plain[r] - _plain_rounded(cfg, w, reqs[r])).max(axis=1)[sorted(per_pos)]
        bound = BF16_GAP_FACTOR * float(np.percentile(gap, 80))
        assert bound < 0.1 * float(np.abs(plain[r]).max()), "the test model is too rough for bfloat16"
        err = np.array([np.abs(row.astype(np.float64) - plain[r][p]).max() for p, row in sorted(per_pos.items())])
        assert err.max() <= BF16_GAP_FACTOR * float(gap.max()), f"{what}: request {r}: position {sorted(per_pos)[int(err.argmax())]}"
        beyond = int((err > bound).sum())
        assert beyond <= max(1, len(err) // 5), (f"{what}: request {r}: {beyond} of {len(err)} positions beyond {bound:.3e}; "
                                                 f"first at {sorted(per_pos)[int(np.argmax(err > bound))]}")


def _poison(cache):
    """Pages and states that nobody holds may contain anything."""
    for g in cache.groups:
        g.k.fill_(float("nan"))
        if g.v is not None:
            g.v.fill_(float("inf"))
    for s in cache.states.values():
        s.fill_(float("nan"))


@pytest.mark.parametrize("case", sorted(lc.CASES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_models_step_like_the_plain_statement_however_the_tokens_are_cut(folders, cuda_device, case, dtype):
    cfg = lc.CASES[case]
    d, w = folders[case, dtype]
    V = cfg["vocab"]
    reqs = {"a": random_tokens(1, 210, V), "b": random_tokens(2, 3, V), "c": random_tokens(3, 77, V), "d": random_tokens(4, 131, V)}
    plain = {r: pl.forward(t, w, cfg) for r, t in reqs.items()}
    model = bn.load_model(d, dtype=dtype)
    cache = model.new_cache(max_tokens=64 * 12, max_seqs=4)
    _poison(cache)
    schedules = (
        ("whole", trace_whole(reqs)),
        ("every token alone", trace_tail({"c": reqs["c"], "b": reqs["b"]}, 1000)),
        ("150 tokens decoded one by one", trace_tail({"a": reqs["a"]}, 150)),
        ("pieces down to two tokens", trace_chunks(reqs, pieces=(2, 1, 5, 64, 33))),
        ("pieces of a page and around it", trace_chunks({"a": reqs["a"], "d": reqs["d"]}, pieces=(63, 1, 64, 65), stagger=2)),
        ("unequal batches, slots and pages used again",
         trace_batches([{"a": (reqs["a"], 40), "b": (reqs["b"], 2), "c": (reqs["c"], 9)},
                        {"d": (reqs["d"], 70), "b": (reqs["b"], 1)}, {"c": (reqs["c"], 76), "a": (reqs["a"], 3)}])),
    )
    for what, steps in schedules:
        _check(replay(model, cache, steps), cfg, w, reqs, plain, dtype, f"case {case}, {what}, {dtype}")
        assert cache.slots.n_free == cache.slots.n_slots
    model.check_kernels()


def test_the_stream_after_every_layer_is_the_plain_statements(folders, cuda_device):
    for case in sorted(lc.CASES):
        cfg = lc.CASES[case]
        d, w = folders[case, "float32"]
        toks = random_tokens(9, 90, cfg["vocab"])
        want = []
        pl.forward(toks, w, cfg, taps=want)
        model = bn.load_model(d, dtype="float32")
        for cut in (90, 60):  # in one step; and the last thirty one by one
            diag = model.diagnostics = bn.Diagnostics(dump_tag="lout", keep=True, out=io.StringIO())
            cache = model.new_cache(max_tokens=256, max_seqs=1)
            slot = cache.open()
            model.step(cache, [bn.SeqStep(slot, toks[:cut], [cut - 1])])
            for tok in toks[cut:]:
                model.step(cache, [bn.SeqStep(slot, [tok], [0])])
            cache.close(slot)
            for i, ref in enumerate(want):
                for pos in (0, 1, 40, 61, 89):
                    (got,) = [r["values"] for r in diag.records if (r["tag"], r["layer"], r["pos"]) == ("lout", i, pos)]
                    assert np.abs(got - ref[pos]).max() < 1e-4 * max(1.0, np.abs(ref[pos]).max()), f"case {case}, after layer {i}, position {pos}"


@pytest.mark.parametrize("case", ["A", "C"])
def test_a_request_alone_and_in_a_batch_give_the_same_logits(folders, cuda_device, case):
    cfg = lc.CASES[case]
    d, _w = folders[case, "float32"]
    V = cfg["vocab"]
    reqs = {"a": random_tokens(11, 100, V), "b": random_tokens(12, 7, V), "c": random_tokens(13, 160, V)}
    model = bn.load_model(d, dtype="float32")
    cache = model.new_cache(max_tokens=64 * 10, max_seqs=3)
    alone = replay(model, cache, trace_whole(reqs))
    together = replay(model, cache, trace_batches([{r: (t, min(12, len(t) - 1)) for r, t in reqs.items()}]))
    for r in reqs:
        for p, row in together[r].items():
            assert np.abs(row - alone[r][p]).max() < 5e-5 * max(1.0, np.abs(row).max()), f"request {r}, position {p}"


@pytest.mark.parametrize("case,dtype", [("C", "float32"), ("C", "bfloat16"), ("A", "bfloat16")])
def test_a_long_prompt_and_long_decoding(folders, cuda_device, case, dtype):
    cfg = lc.CASES[case]
    d, w = folders[case, dtype]
    toks = random_tokens(17, 1400, cfg["vocab"])
    plain = {"x": pl.forward(toks, w, cfg)}
    model = bn.load_model(d, dtype=dtype)
    cache = model.new_cache(max_tokens=1536, max_seqs=1)
    _poison(cache)
    steps = trace_tail({"x": toks}, 300)
    # of the prompt, logits at the edges of pages and pieces and at its end only, to keep the test quick
    steps[0]["entries"][0]["want"] = [0, 1, 2, 63, 64, 65, 127, 128, 511, 512, 1023, 1024, 1099]
    _check(replay(model, cache, steps), cfg, w, {"x": toks}, plain, dtype, f"1,100 tokens and 300 more one by one, {dtype}")
    assert cache.slots.n_free == cache.slots.n_slots


EDGES = {
    "one of everything": [
        {"type": "parallel", "mixer": lc.pair(1, 1, 8, 8, 1, 2, 10.0, None, 0.7, 8, 1, 1, 1.0, 1.0), "mlp": lc.moe(1, 0, 1, 1, 1, 8, 8)},
        {"type": "lightning", "mixer": {"heads": 1, "dim": 8, "vdim": 8, "decay": [1.0]}, "mlp": None},
        {"type": "latent_attention", "mixer": lc.latent(1, 8, 2, 8, 8, 8, 0.7, 10.0), "mlp": None}],
    "many taps, blocks of one channel, a window beyond the sequence": [
        {"type": "parallel", "mixer": lc.pair(4, 2, 16, 16, 5000, 16, 100.0, 32.0, 0.3, 24, 24, 16, 0.3, -2.0), "mlp": lc.moe(3, 3, 2, 6, 5, 3, 8)},
        {"type": "parallel", "mixer": lc.pair(2, 1, 4, 12, 2, 4, 7.0, 0.5, 0.9, 20, 2, 9), "mlp": lc.moe(2, 6, 4, 2, 1, 16, 8)}],
    "recurrences only, decays of none and all": [
        {"type": "lightning", "mixer": {"heads": 2, "dim": 16, "vdim": 40, "decay": [0.0, 1.0]}, "mlp": None},
        {"type": "lightning", "mixer": {"heads": 3, "dim": 160, "vdim": 4, "decay": [0.9, 0.0, 0.99]}, "mlp": None}],
    "three readers of one layer's rows": [
        {"type": "latent_attention", "mixer": lc.latent(8, 4, 4, 12, 8, 12, 0.9, 100.0), "mlp": lc.moe(4, 1, 1, 5, 1, 24, 8)},
        *[{"type": "latent_attention", "mixer": lc.latent(h, d, 4, v, q, 12, 0.6, 100.0, kv_from=0), "mlp": None} for h, d, v, q in ((1, 20, 7, 5), (2, 16, 16, 40), (5, 4, 4, 8))]],
    "all experts for every token, and forty narrow ones": [
        {"type": "lightning", "mixer": {"heads": 8, "dim": 4, "vdim": 12, "decay": [0.9] * 8}, "mlp": lc.moe(5, 1, 6, 1, 1, 12, 300)},
        {"type": "latent_attention", "mixer": lc.latent(2, 32, 32, 32, 300, 224, 0.2, 1e4), "mlp": lc.moe(36, 4, 8, 10, 3, 4, 4)}],
}


@pytest.mark.parametrize("kind", sorted(EDGES))
def test_models_at_the_edges_of_what_the_configuration_allows(tmp_path, cuda_device, kind):
    cfg = {"architecture": "Lakadra", "vocab": 53, "width": 32, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "logit_softcap": 50.0, "layers": EDGES[kind]}
    reqs = {"a": random_tokens(1, 140, 53), "b": random_tokens(2, 1, 53), "c": random_tokens(3, 66, 53)}
    for dtype in ("float32", "bfloat16"):
        w = lc.draw_weights(cfg, seed=8, calm=dtype == "bfloat16")
        d = lc.write_folder(str(tmp_path / dtype), cfg, w)
        plain = {r: pl.forward(t, w, cfg) for r, t in reqs.items()}
        model = bn.load_model(d, dtype=dtype)
        cache = model.new_cache(max_tokens=64 * 8, max_seqs=3)
        _poison(cache)
        for what, steps in (("whole", trace_whole(reqs)), ("pieces", trace_chunks(reqs, pieces=(2, 31, 1, 64))),
                            ("batch", trace_batches([{"a": (reqs["a"], 30), "b": (reqs["b"], 0), "c": (reqs["c"], 65)}]))):
            _check(replay(model, cache, steps), cfg, w, reqs, plain, dtype, f"{kind}, {what}, {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wider_model(tmp_path, cuda_device, dtype):
    """Rows of a thousand numbers (norms on clusters of blocks), heads of 128, key rows of a latent layer beyond 256 numbers."""
    cfg = {"architecture": "Lakadra", "vocab": 200, "width": 1024, "norm": {"eps": 1e-6}, "logit_scale": 0.6, "logit_softcap": 15.0, "layers": [
        {"type": "lightning", "mixer": {"heads": 4, "dim": 128, "vdim": 128, "decay": [0.9, 0.99, 0.999, 0.9999]}, "mlp": lc.moe(6, 2, 2, 4, 2, 256, 512)},
        {"type": "latent_attention", "mixer": lc.latent(4, 128, 64, 128, 256, 512, 0.05, 1e6), "mlp": lc.moe(4, 0, 2, 2, 2, 320, 128)},
        {"type": "parallel", "mixer": lc.pair(8, 2, 128, 64, 90, 64, 1e5, 8.0, 0.06, 1024, 8, 4), "mlp": lc.moe(3, 1, 1, 1, 1, 160, 256)},
        {"type": "latent_attention", "mixer": lc.latent(8, 64, 64, 64, 128, 512, 0.06, 1e6, kv_from=1), "mlp": None}]}
    w = lc.draw_weights(cfg, seed=12, calm=dtype == "bfloat16")
    d = lc.write_folder(str(tmp_path / "m"), cfg, w)
    reqs = {"a": random_tokens(5, 200, 200), "b": random_tokens(6, 40, 200)}
    plain = {r: pl.forward(t, w, cfg) for r, t in reqs.items()}
    model = bn.load_model(d, dtype=dtype)
    cache = model.new_cache(max_tokens=64 * 8, max_seqs=2)
    _poison(cache)
    for what, steps in (("whole", trace_whole(reqs)), ("pieces", trace_chunks(reqs, pieces=(70, 1, 33))),
                        ("batch", trace_batches([{"a": (reqs["a"], 20), "b": (reqs["b"], 8)}]))):
        _check(replay(model, cache, steps), cfg, w, reqs, plain, dtype, f"wider model, {what}, {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point_and_the_replay_program(folders, cuda_device, tmp_path, dtype):
    cfg = lc.CASE_A
    d, w = folders["A", dtype]
    V = cfg["vocab"]
    model = bn.load_model(d, dtype=dtype)
    assert model.graph_safe()  # decode steps are recorded and replayed
    prompts = [random_tokens(31, 50, V), random_tokens(32, 3, V), random_tokens(33, 120, V)]
    got = bn.generate(model, prompts, max_new_tokens=[70, 20, 24])
    for p, g in zip(prompts, got):
        assert len(g.tokens) in (70, 20, 24) and g.finish_reason == "length"
        seq = list(p) + g.tokens[:-1]
        ref = pl.forward(seq, w, cfg)[len(p) - 1:]
        if dtype == "float32":
            slack = 2 * TOL_F32 * max(1.0, float(np.abs(ref).max()))
        else:
            slack = 2 * BF16_GAP_FACTOR * float(np.abs(pl.forward(seq, w, cfg, r=pl.to_bf16)[len(p) - 1:] - ref).max())
        off = [i for i, t in enumerate(g.tokens) if ref[i, t] < ref[i].max() - slack]
        assert not off, f"tokens {off[:5]} of a prompt of {len(p)} are not the plain statement's"
    # a second call on the same model: slots, pages and states are used again
    again = bn.generate(model, prompts[::-1], max_new_tokens=[24, 20, 70])
    assert [g.tokens for g in again[::-1]] == [g.tokens for g in got]
    reqs = {"x": prompts[0] + got[0].tokens, "y": prompts[1]}
    steps = trace_tail(reqs, 6)
    out = str(tmp_path / "out")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", out,
                        "--max-tokens", "256"], input=steps_to_jsonl(steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    plain = {k: pl.forward(t, w, cfg) for k, t in reqs.items()}
    _check(collect_trace_output(steps, out, V), cfg, w, reqs, plain, dtype, "through bin/trace_run")


def test_the_command_line_writes_a_random_model_of_the_design_and_generates_from_it(tmp_path, cuda_device):
    cfgp = tmp_path / "cfg.json"
    cfgp.write_text(json.dumps(lc.CASE_C))
    folder = tmp_path / "m"
    cmd = [sys.executable, os.path.join(ROOT, "bin", "bitnet"), str(folder), "--random-weights", "--config", str(cfgp),
           "--weight-seed", "3", "--dtype", "float32", "--prompt-token-ids", "5,17,3,9,9,1", "--prompt-token-ids", "7",
           "-n", "9", "--repeat-penalty", "1.0", "--token-ids"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    lines = [[int(t) for t in l.split(",")] for l in p.stdout.splitlines() if l.strip()]
    assert [len(l) for l in lines] == [9, 9] and "Generation complete tokens=18" in p.stderr

"""The Rudolix design on the GPU against its plain statement (tests/plain_rudolix.py): every kernel it brought or
extended alone, then whole models of small sizes (tests/rudolix_cases.py) through the step function, the cache and its
states, the generation loop and the replay program."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import bitnet_c_b200 as bn
import plain_rudolix as pr
import rudolix_cases as rc
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
bf = pr.to_bf16
f32 = lambda a: np.asarray(a, dtype=np.float32).astype(np.float64)


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).to("cuda", dtype)


def ints(a):
    return torch.tensor(list(a), dtype=torch.int32, device="cuda")


# ---- kernels alone -----------------------------------------------------------------------------------
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 7, 16])
@pytest.mark.parametrize("width", [50, 96, 1032, 2048])
def test_streams_are_updated_read_and_normed_in_one_pass(cuda_device, streams, width):
    """With and without an update, a layer scale, a bias; every row, or some rows with the streams left alone; a mean far
    from zero; rows of whole 16-byte pieces or not, few rows of wide models (clusters of blocks) or many."""
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(streams * 10000 + width)
    S, W, m, eps = streams, width, 0.7, 1e-5
    for n, dtype in ((5, "float32"), (300, "bfloat16"), (7, "bfloat16")):
        t = DT[dtype]
        xs = f32(rng.standard_normal((S, n, W)) + 20.0)  # the mean dwarfs the spread
        y, ls = bf(rng.standard_normal((n, W))), f32(1 + 0.3 * rng.standard_normal(W))
        mix, out, read = f32(rng.standard_normal((S, S)) / S), f32(rng.standard_normal(S)), f32(rng.standard_normal(S) / S)
        w, b = bf(1 + 0.3 * rng.standard_normal(W)), bf(rng.standard_normal(W))
        x = dev(xs.transpose(1, 0, 2).reshape(n, S * W))
        coef = dev(np.concatenate([mix.ravel(), out]))
        new = pr.update_streams(xs, mix, out, m, y * ls)
        tol = 3e-4 if dtype == "float32" else 2.0 ** -6  # rows with means of twenty and spreads of about one
        rows = [n - 1, 0, 2]
        some = ops.streams_norm(x, S, dev(w, t), dev(b, t), eps, t, delta=dev(y, t), mix=coef, scale=dev(ls), mult=m, read=dev(read), rows=ints(rows))
        assert torch.equal(x, dev(xs.transpose(1, 0, 2).reshape(n, S * W)))  # with rows the streams stay as they are
        h = ops.streams_norm(x, S, dev(w, t), dev(b, t), eps, t, delta=dev(y, t), mix=coef, scale=dev(ls), mult=m, read=dev(read))
        got = x.cpu().numpy().reshape(n, S, W).transpose(1, 0, 2)
        assert np.abs(got - new).max() < 2e-6 * np.abs(xs).sum(0).max()
        want = pr.layer_norm(pr.read_streams(new, read), w, b, eps)
        assert np.abs(h.float().cpu().numpy() - want).max() < tol * np.abs(want).max()
        assert np.abs(some.float().cpu().numpy() - want[rows]).max() < tol * np.abs(want).max()
        plain = ops.streams_norm(x, S, dev(w, t), None, eps, torch.float32)  # no update, no bias, the streams' plain sum
        assert np.abs(plain.cpu().numpy() - pr.layer_norm(got.astype(np.float64).sum(0), w, 0.0, eps)).max() < 3e-3
    if S == 1:  # one stream without a matrix is an ordinary residual sum
        x = dev(xs[0])
        h = ops.streams_norm(x, 1, dev(w), dev(b), eps, torch.float32, delta=dev(y), mult=1.0)
        assert np.abs(x.cpu().numpy() - (xs[0] + y)).max() < 1e-5
        assert np.abs(h.cpu().numpy() - pr.layer_norm(xs[0] + y, w, b, eps)).max() < 3e-4


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 9, 16])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [50, 64, 1024])
def test_the_input_convolution_however_the_tokens_are_cut(cuda_device, taps, dtype, width):
    """Three sequences in scattered slots, in steps of runs down to two tokens (and one token beside them) and in steps
    of one token for all, taken inside the norm's pass: the same rows as the convolution of the whole sequence; a slot
    that is in no step keeps what it holds."""
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(taps * 100 + width)
    t = DT[dtype]
    lens, slots = [40, 33, 28], [4, 0, 2]
    w, b = bf(1 + 0.3 * rng.standard_normal(width)), bf(rng.standard_normal(width))
    conv = bf(rng.standard_normal((width, taps)) * 0.6)
    x = [f32(rng.standard_normal((n, width))) for n in lens]
    rnd = bf if dtype == "bfloat16" else (lambda a: a)
    h = [rnd(pr.layer_norm(a, w, b, 1e-5)) for a in x]
    want = [a + pr.causal_convolution(a, conv) for a in h]
    hist = torch.zeros((5, max(taps - 1, 0), width), dtype=t, device="cuda") if taps > 1 else None
    if hist is not None:
        hist[1].fill_(7.0)
    wd, bd, td = dev(w, t), dev(b, t), dev(conv.T.copy())
    at = [0, 0, 0]
    scale = max(np.abs(a).max() for a in want)
    for new in ([7, 1, 2], [2, 2, 2], [1, 1, 1], [3, 1, 5], [1, 1, 1], [1, 1, 1], [17, 2, 1], [2, 20, 2], [1, 1, 1], [5, 3, 12]):
        rows = np.concatenate([x[s][at[s]:at[s] + c] for s, c in enumerate(new)])
        ref = np.concatenate([want[s][at[s]:at[s] + c] for s, c in enumerate(new)])
        xd = dev(rows)
        if max(new) == 1:
            got = ops.streams_norm(xd, 1, wd, bd, 1e-5, t, taps=td, hist=hist, slots=ints(slots))
        else:
            normed = ops.streams_norm(xd, 1, wd, bd, 1e-5, t)
            seq = np.concatenate([np.full(c, s) for s, c in enumerate(new)])
            got = ops.input_convolution(normed, td, hist, ints(seq), ints(np.concatenate([[0], np.cumsum(new)])), ints(slots))
        err = np.abs(got.float().cpu().numpy() - ref).max()
        assert err < (1e-5 if dtype == "float32" else 2.0 ** -6) * max(1.0, scale), f"step {new} from {at}: {err:.3e}"
        at = [a + c for a, c in zip(at, new)]
    assert at == lens
    if hist is not None:
        assert bool((hist[1] == 7.0).all()) and bool((hist[3] == 0.0).all())


STATE_SHAPES = [  # heads, groups, state rows, value width, taps
    (4, 2, 16, 24, 4), (1, 1, 40, 136, 2), (2, 1, 10, 7, 1), (2, 2, 132, 40, 3), (3, 3, 256, 8, 16), (6, 2, 64, 64, 4), (5, 1, 6, 33, 5),
    (8, 1, 128, 64, 4),
]


def _state_inputs(rng, T, shape, delta, decay):
    H, G, d, dv, taps = shape
    n_qk, n_v = G * d, H * dv
    lo, hi = {"mixed": (-4.0, 1.0), "slow": (-9.0, -8.0), "fast": (2.0, 3.0)}[decay]
    return {"q": bf(rng.standard_normal((T, n_qk))), "k": bf(rng.standard_normal((T, n_qk))), "v": bf(rng.standard_normal((T, n_v))),
            "a": f32(rng.standard_normal((T, H))), "b": f32(rng.standard_normal((T, H))),
            "conv": f32(rng.standard_normal((2 * n_qk + n_v, taps)) * 0.7), "bias": None if delta else f32(0.3 * rng.standard_normal(2 * n_qk + n_v)),
            "dt_bias": f32(rng.standard_normal(H) - 1), "a_log": f32(rng.uniform(lo, hi, H)), "d": None if delta else f32(rng.standard_normal(H))}


def _plain_state(z, shape, delta):
    """One sequence through the plain functions: [T, heads * vdim]."""
    H, G, d, dv, _taps = shape
    T, n_qk = z["q"].shape[0], G * d
    part = lambda lo, hi: None if z["bias"] is None else z["bias"][lo:hi]
    q = pr.silu(pr.causal_convolution(z["q"], z["conv"][:n_qk], part(0, n_qk))).reshape(T, G, d)
    k = pr.silu(pr.causal_convolution(z["k"], z["conv"][n_qk:2 * n_qk], part(n_qk, 2 * n_qk))).reshape(T, G, d)
    v = pr.silu(pr.causal_convolution(z["v"], z["conv"][2 * n_qk:], part(2 * n_qk, None))).reshape(T, H, dv)
    step = pr.softplus(z["a"] + z["dt_bias"])
    out = np.zeros((T, H, dv))
    if delta:
        q, k = pr.unit_vector(q) * d ** -0.5, pr.unit_vector(k)
    for h in range(H):
        g = pr.shared_head(h, H, G)
        if delta:
            out[:, h] = pr.delta_rule(q[:, g], k[:, g], v[:, h], np.exp(-np.exp(z["a_log"][h]) * step[:, h]), pr.sigmoid(z["b"][:, h]))[0]
        else:
            out[:, h] = pr.state_space(v[:, h], k[:, g], q[:, g], step[:, h], float(np.exp(z["a_log"][h])), float(z["d"][h]))[0]
    return out.reshape(T, H * dv)


def _run_state(zs, shape, delta, steps, dtype, slots, state, chunks):
    """The kernel over ``steps`` (new tokens per sequence); returns the sequences' outputs."""
    from bitnet_c_b200.csrc import ops
    H, G, d, dv, taps = shape
    n_qk, n_v = G * d, H * dv
    z0 = zs[0]
    conv, one = dev(z0["conv"].T.copy()), lambda k: None if z0[k] is None else dev(z0[k])
    at, got = [0] * len(zs), [np.zeros((z["q"].shape[0], n_v), dtype=np.float32) for z in zs]
    for new in steps:
        live = [s for s, c in enumerate(new) if c]
        cat = lambda k: np.concatenate([zs[s][k][at[s]:at[s] + new[s]] for s in live])
        # rows as a mixer's product leaves them: values first, something else, keys, queries, the gates behind
        between = np.full((sum(new), 4), 1e3)
        proj = dev(np.concatenate([cat("v"), between, cat("k"), cat("q")], axis=1), DT[dtype])
        gates = dev(np.concatenate([cat("a"), cat("b")], axis=1))
        counts = [new[s] for s in live]
        tiles = [(i, r) for i, c in enumerate(counts) for r in range(0, c, 64)]
        kw = dict(tile_seq=ints(i for i, _ in tiles), tile_row0=ints(r for _, r in tiles)) if chunks else {}
        o = ops.gated_state(proj, n_v + 4 + n_qk, n_v + 4, 0, gates, 0, H if delta else -1, conv, one("bias"), one("dt_bias"), one("a_log"),
                            one("d"), state, ints(np.concatenate([np.full(c, i) for i, c in enumerate(counts)])),
                            ints(np.concatenate([[0], np.cumsum(counts)])), ints([at[s] for s in live]), ints([slots[s] for s in live]),
                            len(live), H, G, d, dv, one_token=max(counts) == 1, **kw).cpu().numpy()
        r = 0
        for s in live:
            got[s][at[s]:at[s] + new[s]] = o[r:r + new[s]]
            r += new[s]
            at[s] += new[s]
    assert at == [len(g) for g in got]
    return got


@pytest.mark.parametrize("shape", STATE_SHAPES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("kind", ["delta", "state space"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_matrix_states_however_the_tokens_are_cut(cuda_device, shape, kind, dtype):
    """Both recurrences over unequal sequences in scattered slots: token by token and chunk by chunk, in runs that end
    before, on and behind the edge of a chunk, in pairs, and one token at a time; slots that are in no step keep what
    they hold."""
    from bitnet_c_b200.csrc import ops
    H, G, d, dv, taps = shape
    delta = kind == "delta"
    rng = np.random.default_rng(H * 1000 + d)
    lens, slots = [150, 4, 67], [3, 0, 4]
    z0 = _state_inputs(rng, 1, shape, delta, "mixed")
    zs = []
    for n in lens:
        z = _state_inputs(rng, n, shape, delta, "mixed")
        z.update({k: z0[k] for k in ("conv", "bias", "dt_bias", "a_log", "d")})
        zs.append(z)
    want = [_plain_state(z, shape, delta) for z in zs]
    scale = max(np.abs(a).max() for a in want)
    plans = {"whole": [[150, 4, 67]],
             "around a chunk's edge": [[63, 1, 64], [1, 0, 1], [65, 1, 0], [21, 2, 2]],
             "pairs and single tokens": [[2, 2, 2], [1, 1, 1], [1, 1, 1], [100, 0, 20], [1, 0, 1], [2, 0, 2], [43, 0, 40]]}
    for what, steps in plans.items():
        for chunks in (False, True):
            if chunks and d % 4:
                continue
            state = torch.zeros((6, ops.gated_state_floats(H, G, d, dv, taps)), dtype=torch.float32, device="cuda")
            state[1].fill_(7.0)
            got = _run_state(zs, shape, delta, steps, dtype, slots, state, chunks)
            for s, (a, b) in enumerate(zip(got, want)):
                err = np.abs(a - b).max(axis=1)
                assert np.isfinite(a).all() and err.max() < 1e-4 * max(1.0, scale), \
                    f"{what}, chunks {chunks}: sequence {s}, token {int(err.argmax())}: {err.max():.3e} of {scale:.2f}"
            assert bool((state[1] == 7.0).all()) and bool((state[2] == 0.0).all())


@pytest.mark.parametrize("kind", ["delta", "state space"])
def test_one_write_among_hundreds_of_tokens_is_read_back_or_forgotten(cuda_device, kind):
    """All values are zero but one token's, planted at the start, just inside and just outside the edges of chunks: with
    slow decays every later read-out holds it, with fast ones hardly any; in one run, in runs that part at the plant,
    and decoded."""
    from bitnet_c_b200.csrc import ops
    shape = (4, 2, 32, 48, 3)
    delta = kind == "delta"
    rng = np.random.default_rng(3)
    n = 300
    for decay in ("slow", "fast"):
        for p in (0, 1, 62, 63, 64, 127, 128, 200):
            z = _state_inputs(rng, n, shape, delta, decay)
            if not delta:
                z["bias"][:] = 0.0
                z["d"][:] = 0.0
            z["v"][:] = 0.0
            z["v"][p] = 50.0
            want = _plain_state(z, shape, delta)
            far = np.abs(want[p + 60:]).max()
            assert (far > 1e-2) if decay == "slow" else (far < 1e-6)
            for steps, chunks in (([[n]], True), ([[n]], False), ([[p + 1], [n - p - 1]], True), ([[40]] + [[1]] * 60 + [[n - 100]], True)):
                state = torch.zeros((1, ops.gated_state_floats(4, 2, 32, 48, 3)), dtype=torch.float32, device="cuda")
                got = _run_state([z], shape, delta, steps, "float32", [0], state, chunks)[0]
                err = np.abs(got - want).max(axis=1)
                assert err.max() < 2e-5 * np.abs(want).max(), f"{decay}, plant {p}, {steps[:3]}, chunks {chunks}: token {int(err.argmax())}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("parts,length", [(4, 24), (1, 7), (3, 33), (1, 200), (2, 1030), (5, 64), (1, 4096)])
def test_gated_norms_behind_a_recurrence(cuda_device, dtype, parts, length):
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(parts * length)
    n, row, t = 19, parts * length, DT[dtype]
    o, z = f32(rng.standard_normal((n, row)) * 3), bf(rng.standard_normal((n, row)) * 2)
    wide = dev(np.concatenate([np.full((n, 8), 9.0), z, np.full((n, 4), 9.0)], axis=1), t)
    for gain_len in {row, length}:
        gain = f32(1 + 0.3 * rng.standard_normal(gain_len))
        g = np.tile(gain, row // gain_len)
        first = pr.grouped_rms(o * pr.silu(z), parts, 1e-5) * g
        last = pr.grouped_rms(o, parts, 1e-5) * g * pr.silu(z)
        for gate_first, want in ((True, first), (False, last)):
            got = ops.state_output(dev(o), wide[:, 8:8 + row], dev(gain), parts, 1e-5, gate_first, t).float().cpu().numpy()
            assert np.abs(got - want).max() < (1e-5 if dtype == "float32" else 2.0 ** -7) * max(1.0, np.abs(want).max())


def test_polynomials_of_normed_powers_and_routers_with_a_bias(cuda_device):
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(4)
    coef = f32([0.7, -0.4, 0.9, 0.3])
    for n, length, row in ((9, 64, 64), (5, 37, 40), (300, 200, 200), (3, 9000, 9000), (2, 1, 8)):
        z = np.full((n, row), 1e4)
        z[:, :length] = bf(rng.standard_normal((n, length)) * 3)
        for zt, ot, tol in ((torch.float32, torch.float32, 1e-5), (torch.float32, torch.bfloat16, 2.0 ** -7), (torch.bfloat16, torch.bfloat16, 2.0 ** -7)):
            got = ops.poly_norm(dev(z, zt), dev(coef), 1e-5, ot, length=length).float().cpu().numpy()
            want = pr.poly_norm(z[:, :length], coef, 1e-5)
            assert np.abs(got[:, :length] - want).max() < tol * max(1.0, np.abs(want).max()) and np.all(got[:, length:] == 0)
    for E, top, width in ((8, 2, 64), (5, 5, 50), (40, 7, 96), (1, 1, 16)):
        h, w, b = bf(rng.standard_normal((33, width))), bf(rng.standard_normal((E, width)) / 8), f32(rng.standard_normal(E) * 2)
        ids, wts = pr.route(h, {"router": w, "router.b": b}, "", top)
        for t in (torch.float32, torch.bfloat16):
            gi, gw = ops.moe_route(dev(h, t), dev(w, t), top, renormalise=True, softmax=True, bias=dev(b))
            assert np.array_equal(gi.cpu().numpy(), ids) and np.abs(gw.cpu().numpy() - wts).max() < 1e-5


def test_embedding_rows_side_by_side(cuda_device):
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(5)
    table = bf(rng.standard_normal((11, 50)))
    bad = torch.zeros(1, dtype=torch.int32, device="cuda")
    out = torch.full((4, 150), float("nan"), device="cuda")
    ops.embed_gather(dev(table), ints([3, 0, 10, 3]), out, bad, 2.5, copies=3)
    assert np.array_equal(out.cpu().numpy(), np.tile((table[[3, 0, 10, 3]] * 2.5).astype(np.float32), (1, 3))) and int(bad) == 0
    ops.embed_gather(dev(table), ints([3, 11, 1, 1]), out, bad, 2.5, copies=3)
    assert int(bad) == 1 and bool((out[1] == 0).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dims,heads,kv,dim,vdim", [(8, 4, 2, 32, 16), (32, 8, 1, 32, 64), (10, 3, 3, 10, 7), (2, 6, 2, 48, 48)])
def test_the_attention_mixer_finds_one_key_far_away(cuda_device, dtype, dims, heads, kv, dim, vdim):
    """A mixer whose keys answer its queries, among three hundred tokens: the last one's score stands out for one token
    far back (at a sequence's start, at both sides of a page's edge), whose value dwarfs the others'; whole, in pieces
    behind cached tokens, decoded, beside other sequences, over a cache poisoned with NaN; a sink with a good part of the
    weight."""
    from bitnet_c_b200.cache import Cache
    from bitnet_c_b200.config import BiasAttentionSpec, RotaryBlendSpec
    from bitnet_c_b200.engine.batch import SeqStep, pack_step
    from bitnet_c_b200.parts import BuildContext, build_part
    t = DT[dtype]
    rng = np.random.default_rng(dims * dim)
    W = 64
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 1.0 / np.sqrt(dim), "rot": {"base": 1e7, "dims": dims}}
    spec = BiasAttentionSpec(width=W, n_heads=heads, n_kv_heads=kv, head_dim=dim, v_head_dim=vdim, scale=m["scale"], sink=True,
                             position=RotaryBlendSpec(dims=dims, base=1e7))
    mixer = build_part("mixer", spec, BuildContext(dtype=t, device=torch.device("cuda:0")))
    wk = bf(rng.standard_normal((kv * dim, W)) / 8)
    w = {"k": wk, "q": np.repeat(wk.reshape(kv, dim, W), heads // kv, axis=0).reshape(heads * dim, W), "v": bf(rng.standard_normal((kv * vdim, W)) / 8),
         "o": bf(rng.standard_normal((W, heads * vdim)) / 8), "sink": bf(rng.standard_normal(heads) + 2)}
    mixer.bind({k: dev(a, t) for k, a in w.items()})
    for far in (0, 63, 64, 130):
        hs = [bf(rng.standard_normal((n, W))) for n in (300, 70, 5)]
        hs[0][far] = bf(hs[0][far] * 6.0)
        hs[0][-1] = hs[0][far]
        want = [pr.mixer_attention(h, w, "", m, 1e-5) for h in hs]
        q = (hs[0][-1:] @ w["q"].T).reshape(1, heads, dim)
        scores = (hs[0] @ w["k"].T).reshape(300, kv, dim)[:, 0] @ q[0, 0] * m["scale"]
        assert scores[far] > 1.3 * np.delete(scores, [far, 299]).max()  # it stands out, rotation aside
        cache = Cache([mixer.cache_request()], [None], [None], 64 * 9, 4096, t, torch.device("cuda:0"), max_seqs=3)
        for g in cache.groups:
            g.k.fill_(float("nan"))
            g.v.fill_(float("inf"))
        for steps in ([[300, 70, 5]], [[64, 69, 3], [66, 1, 1], [170, 0, 1]], [[290, 60, 1]] + [[1, 1, 1]] * 4 + [[6, 6, 0]]):
            slots, at = [cache.open() for _ in hs], [0, 0, 0]
            for new in steps:
                live = [s for s in range(3) if new[s]]
                for s in live:
                    cache.reserve(slots[s], new[s])
                cache.sync()
                ctx = pack_step([SeqStep(slots[s], [0] * new[s]) for s in live], [at[s] for s in live], torch.device("cuda:0"))
                rows = np.concatenate([hs[s][at[s]:at[s] + new[s]] for s in live])
                got = mixer.forward(dev(rows, t), ctx, cache.view(0), None).float().cpu().numpy()
                ref = np.concatenate([want[s][at[s]:at[s] + new[s]] for s in live])
                err = np.abs(got - ref).max(axis=1)
                assert np.isfinite(got).all() and err.max() < (2e-5 if dtype == "float32" else 0.03) * max(1.0, np.abs(ref).max()), \
                    f"far {far}, step {new}: row {int(err.argmax())}"
                for s in live:
                    cache.advance(slots[s], new[s])
                    at[s] += new[s]
            for s in slots:
                cache.close(s)


@pytest.mark.parametrize("H,G,d,dv,window", [(4, 2, 32, 16, 0), (8, 1, 128, 128, 0), (3, 3, 48, 80, 0), (16, 4, 64, 64, 70), (2, 1, 112, 32, 129), (6, 2, 16, 128, 1)])
def test_runs_of_tokens_on_tcgen05_with_precise_weights_and_a_sink(cuda_device, H, G, d, dv, window):
    """Whole prompts and pieces behind cached tokens in scattered pages: keys planted just inside and outside a window or at
    the start, values that dwarf the rest, sinks that hold a good part of the weight or exceed every score by far; the
    weights carry 16 bits of mantissa (with weights of 8 bits the result is visibly rougher)."""
    from bitnet_c_b200.csrc import ops
    rng = np.random.default_rng(H * d + window)
    lens = [300, 70, 17]
    T, scale, per = sum(lens), 1.0 / np.sqrt(d), H // G
    q, k, v = (bf(rng.standard_normal((T, n, w))) for n, w in ((H, d), (G, d), (G, dv)))
    last = lens[0] - 1
    far = last - window + 1 if window else 0
    k[far] = bf(q[last].reshape(G, per, d)[:, 0] * 2.0)
    v[far] = bf(8.0 + 0.03 * rng.standard_normal((G, dv)))
    if window:
        k[far - 1], v[far - 1] = bf(q[last].reshape(G, per, d)[:, 0] * 4.0), 500.0  # must not be seen
    starts = np.concatenate([[0], np.cumsum(lens)])
    pages = [(n + 63) // 64 for n in lens]
    order = rng.permutation(sum(pages) + 2)
    table = np.zeros((4, max(pages)), dtype=np.int32)
    kc = torch.full((sum(pages) + 2, G, 64, d), float("nan"), dtype=torch.bfloat16, device="cuda")
    vc = torch.full((sum(pages) + 2, G, 64, dv), float("inf"), dtype=torch.bfloat16, device="cuda")
    at = 0
    for s, n in enumerate(lens):
        table[s + 1, :pages[s]] = order[at:at + pages[s]]
        at += pages[s]
        for p in range(n):
            kc[int(table[s + 1, p // 64]), :, p % 64] = dev(k[starts[s] + p], torch.bfloat16)
            vc[int(table[s + 1, p // 64]), :, p % 64] = dev(v[starts[s] + p], torch.bfloat16)
    table = torch.from_numpy(table).cuda()
    for sink in (None, f32(rng.standard_normal(H) + 3), np.full(H, 200.0)):
        want = np.zeros((T, H, dv))
        for s, n in enumerate(lens):
            i, j = np.arange(n)[:, None], np.arange(n)[None, :]
            seen = (j <= i) & ((i - j < window) if window else True)
            for h in range(H):
                a = slice(starts[s], starts[s] + n)
                sc = np.where(seen, q[a, h] @ k[a, h // per].T * scale, -np.inf)
                want[a, h] = pr.softmax_with_sink(sc, -1e30 if sink is None else float(sink[h])) @ v[a, h // per]
        want = want.reshape(T, H * dv)
        for new in (lens, [150, 33, 16], [129, 2, 1]):
            rows = np.concatenate([np.arange(starts[s] + lens[s] - c, starts[s] + lens[s]) for s, c in enumerate(new)])
            tiles = [(s, r) for s, c in enumerate(new) for r in range(0, c, 128)]
            qd = dev(q.reshape(T, -1)[rows], torch.bfloat16)
            err = {}
            for precise in (True, False):
                out = torch.full((len(rows), H * dv), float("nan"), dtype=torch.bfloat16, device="cuda")
                ops.attention_prefill_tc(qd, H * d, out, H, G, d, scale, window, ints(s for s, _ in tiles), ints(r for _, r in tiles),
                                         ints(np.concatenate([[0], np.cumsum(new)])), ints(n - c for n, c in zip(lens, new)), ints([1, 2, 3]),
                                         table, kc, vc, precise=precise, sink=dev(sink) if sink is not None else None)
                got = out.float().cpu().numpy()
                assert np.isfinite(got).all()
                err[precise] = np.abs(got - want[rows])
            # what is left is the rounding of the result itself
            assert (err[True] <= 2.0 ** -8 * np.abs(want[rows]) + 2e-5 * (1 + np.abs(v).max(where=np.abs(v) < 100, initial=0))).all(), (sink, new)
            assert err[True].sum() < err[False].sum() or window == 1 or (sink is not None and sink[0] == 200.0)
    ops.check_tc_status(torch.device("cuda:0"))


@pytest.mark.parametrize("d", [64, 128])
def test_every_row_of_long_runs_holds_its_last_page(cuda_device, d):
    """A thousand tokens and some, several heads, scores of every temper (warps of a block then run through their rows at
    unequal speeds): the tcgen05 kernel against the general one, row by row."""
    from bitnet_c_b200.csrc import ops
    for seed, n in enumerate((1122, 439, 640, 65, 129, 1000, 770, 1500)):
        H, G = 8, 4
        g = torch.Generator(device="cuda").manual_seed(seed)
        q = (torch.randn((n, H * d), device="cuda", generator=g) * (1 + 3 * (seed % 3))).bfloat16()
        pages = (n + 63) // 64
        k = torch.randn((pages, G, 64, d), device="cuda", generator=g).bfloat16()
        v = torch.randn((pages, G, 64, d), device="cuda", generator=g).bfloat16()
        table = torch.randperm(pages, device="cuda", generator=g).int().view(1, pages)
        sink = torch.randn(H, device="cuda", generator=g) * 2 + 3
        out, ref = (torch.full((n, H * d), float("nan"), dtype=torch.bfloat16, device="cuda") for _ in range(2))
        zero, pos = ints([0]), torch.arange(n, dtype=torch.int32, device="cuda")
        ops.attention_general(q, H * d, ref, n, H, G, d, d ** -0.5, 0, torch.zeros_like(pos), pos, zero, table, k, v, sink=sink)
        tiles = list(range(0, n, 128))
        for precise in (True, False):
            for _ in range(4):
                ops.attention_prefill_tc(q, H * d, out, H, G, d, d ** -0.5, 0, ints([0] * len(tiles)), ints(tiles), ints([0, n]), zero, zero, table,
                                         k, v, precise=precise, sink=sink)
                err = (out.float() - ref.float()).abs().amax(1)
                assert float(err.max()) < 0.05 * float(ref.float().abs().max()), f"{n} tokens, precise {precise}: row {int(err.argmax())}"


# ---- whole models --------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """Per case and number format: (folder, weights).  bfloat16 models have routers whose choices rounding leaves alone."""
    out = {}
    for name, cfg in rc.CASES.items():
        for dtype, calm in (("float32", False), ("bfloat16", True)):
            w = rc.draw_weights(cfg, seed=26, calm=calm)
            out[name, dtype] = (rc.write_folder(str(tmp_path_factory.mktemp("rudolix") / (name + dtype)), cfg, w), w)
    return out


_ROUNDED = {}


def _plain_rounded(cfg, w, tokens):
    key = (json.dumps(cfg, sort_keys=True), id(w), tuple(tokens))
    if key not in _ROUNDED:
        _ROUNDED[key] = pr.forward(tokens, w, cfg, r=pr.to_bf16)
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


@pytest.mark.parametrize("case", sorted(rc.CASES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_models_step_like_the_plain_statement_however_the_tokens_are_cut(folders, cuda_device, case, dtype):
    cfg = rc.CASES[case]
    d, w = folders[case, dtype]
    V = cfg["vocab"]
    reqs = {"a": random_tokens(1, 210, V), "b": random_tokens(2, 3, V), "c": random_tokens(3, 77, V), "d": random_tokens(4, 131, V)}
    plain = {r: pr.forward(t, w, cfg) for r, t in reqs.items()}
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


def test_the_sum_of_streams_after_every_layer_is_the_plain_statements(folders, cuda_device):
    for case in sorted(rc.CASES):
        cfg = rc.CASES[case]
        d, w = folders[case, "float32"]
        toks = random_tokens(9, 90, cfg["vocab"])
        want = []
        pr.forward(toks, w, cfg, taps=want)
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
    cfg = rc.CASES[case]
    d, _w = folders[case, "float32"]
    V = cfg["vocab"]
    reqs = {"a": random_tokens(11, 100, V), "b": random_tokens(12, 7, V), "c": random_tokens(13, 160, V)}
    model = bn.load_model(d, dtype="float32")
    cache = model.new_cache(max_tokens=64 * 10, max_seqs=3)
    alone = replay(model, cache, trace_whole(reqs))
    together = replay(model, cache, trace_batches([{r: (t, min(12, len(t) - 1)) for r, t in reqs.items()}]))
    for r in reqs:
        for p, row in together[r].items():
            assert np.abs(row - alone[r][p]).max() < 2e-5 * max(1.0, np.abs(row).max()), f"request {r}, position {p}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_and_long_decoding(folders, cuda_device, dtype):
    cfg = rc.CASE_C
    d, w = folders["C", dtype]
    toks = random_tokens(17, 1400, cfg["vocab"])
    plain = {"x": pr.forward(toks, w, cfg)}
    model = bn.load_model(d, dtype=dtype)
    cache = model.new_cache(max_tokens=1536, max_seqs=1)
    _poison(cache)
    steps = trace_tail({"x": toks}, 300)
    # of the prompt, logits at the edges of pages and chunks and at its end only, to keep the test quick
    steps[0]["entries"][0]["want"] = [0, 1, 2, 63, 64, 65, 127, 128, 511, 512, 1023, 1024, 1099]
    _check(replay(model, cache, steps), cfg, w, {"x": toks}, plain, dtype, f"1,100 tokens and 300 more one by one, {dtype}")
    assert cache.slots.n_free == cache.slots.n_slots


EDGES = {
    "one head, one expert, one tap, one stream": (dict(streams=1, canon={"taps": 1}), [
        {"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.7, "rot": {"base": 10.0, "dims": 2}},
         "mlp": {"kind": "moe", "router": {"experts": 1, "top": 1}, "expert": {"ff": 8, "limit": 1.0}}},
        {"type": "delta", "mixer": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "conv": 1}, "mlp": None},
        {"type": "mamba2", "mixer": {"heads": 1, "groups": 1, "state": 8, "vdim": 8, "conv": 1, "norm_groups": 1}, "mlp": None}]),
    "many taps and streams": (dict(streams=6, canon={"taps": 11}, residual_mult=0.3), [
        {"type": "mamba2", "mixer": {"heads": 4, "groups": 4, "state": 4, "vdim": 4, "conv": 16, "norm_groups": 8}, "mlp": {"kind": "dense", "ff": 8}},
        {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 4, "vdim": 4, "conv": 9}, "mlp": {"kind": "dense", "ff": 3}}]),
    "recurrences only, no feed-forward": (dict(streams=2, canon={"taps": 3}), [
        {"type": "delta", "mixer": {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 40, "conv": 4}, "mlp": None},
        {"type": "mamba2", "mixer": {"heads": 2, "groups": 1, "state": 16, "vdim": 40, "conv": 4, "norm_groups": 2}, "mlp": None}]),
    "attention only": (dict(streams=3, canon={"taps": 2}), [
        {"type": "attention", "mixer": {"heads": 8, "kv_heads": 1, "dim": 4, "vdim": 12, "scale": 0.9, "rot": {"base": 100.0, "dims": 4}},
         "mlp": {"kind": "dense", "ff": 24}}] * 3),
    "all experts for every token, narrow and wide": (dict(streams=2, canon={"taps": 3}), [
        {"type": "delta", "mixer": {"heads": 8, "kv_heads": 8, "dim": 4, "vdim": 12, "conv": 2},
         "mlp": {"kind": "moe", "router": {"experts": 6, "top": 6}, "expert": {"ff": 12, "limit": 0.5}}},
        {"type": "delta", "mixer": {"heads": 1, "kv_heads": 1, "dim": 160, "vdim": 4, "conv": 2},
         "mlp": {"kind": "moe", "router": {"experts": 40, "top": 1}, "expert": {"ff": 100, "limit": 7.0}}}]),
}


@pytest.mark.parametrize("kind", sorted(EDGES))
def test_models_at_the_edges_of_what_the_configuration_allows(tmp_path, cuda_device, kind):
    top, layers = EDGES[kind]
    cfg = {"architecture": "Rudolix", "vocab": 53, "width": 32, "residual_mult": 0.5, "norm": {"eps": 1e-6}, "embedding": {"scale": 4.0},
           **top, "layers": layers}
    reqs = {"a": random_tokens(1, 140, 53), "b": random_tokens(2, 1, 53), "c": random_tokens(3, 66, 53)}
    for dtype in ("float32", "bfloat16"):
        w = rc.draw_weights(cfg, seed=8, calm=dtype == "bfloat16")
        d = rc.write_folder(str(tmp_path / dtype), cfg, w)
        plain = {r: pr.forward(t, w, cfg) for r, t in reqs.items()}
        model = bn.load_model(d, dtype=dtype)
        cache = model.new_cache(max_tokens=64 * 8, max_seqs=3)
        _poison(cache)
        for what, steps in (("whole", trace_whole(reqs)), ("pieces", trace_chunks(reqs, pieces=(2, 31, 1, 64))),
                            ("batch", trace_batches([{"a": (reqs["a"], 30), "b": (reqs["b"], 0), "c": (reqs["c"], 65)}]))):
            _check(replay(model, cache, steps), cfg, w, reqs, plain, dtype, f"{kind}, {what}, {dtype}")


def test_tensors_of_a_sublayer_that_is_left_out_are_read_past(tmp_path, cuda_device):
    cfg = rc.CASE_B
    w = rc.draw_weights(cfg, seed=3)
    full = {**cfg, "layers": [{**l, "mlp": l["mlp"] or {"kind": "dense", "ff": 8}} for l in cfg["layers"]]}
    spare = {n: a for n, a in rc.draw_weights(full, seed=4).items() if n not in w and ".mlp." not in n}
    assert len(spare) == 7
    toks = random_tokens(1, 40, cfg["vocab"])
    logits = []
    for k, tensors in (("a", w), ("b", {**w, **spare})):
        model = bn.load_model(rc.write_folder(str(tmp_path / k), cfg, tensors), dtype="float32")
        cache = model.new_cache(max_tokens=64, max_seqs=1)
        logits.append(model.step(cache, [bn.SeqStep(cache.open(), toks, [39])]))
    assert torch.equal(*logits)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wider_model(tmp_path, cuda_device, dtype):
    """Rows of a thousand numbers (norms on clusters of blocks), heads of 128, states of 128 x 64, groups shared by many heads."""
    cfg = {"architecture": "Rudolix", "vocab": 200, "width": 1024, "streams": 2, "residual_mult": 0.5, "norm": {"eps": 1e-6},
           "canon": {"taps": 4}, "embedding": {"scale": 1.0}, "layers": [
               {"type": "mamba2", "mixer": {"heads": 8, "groups": 1, "state": 128, "vdim": 64, "conv": 4, "norm_groups": 1}, "mlp": {"kind": "dense", "ff": 1500}},
               {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 128, "vdim": 128, "conv": 4},
                "mlp": {"kind": "moe", "router": {"experts": 4, "top": 2}, "expert": {"ff": 160, "limit": 2.0}}},
               {"type": "attention", "mixer": {"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 64, "scale": 0.05, "rot": {"base": 1e6, "dims": 64}},
                "mlp": None}]}
    w = rc.draw_weights(cfg, seed=12, calm=dtype == "bfloat16")
    d = rc.write_folder(str(tmp_path / "m"), cfg, w)
    reqs = {"a": random_tokens(5, 200, 200), "b": random_tokens(6, 40, 200)}
    plain = {r: pr.forward(t, w, cfg) for r, t in reqs.items()}
    model = bn.load_model(d, dtype=dtype)
    cache = model.new_cache(max_tokens=64 * 8, max_seqs=2)
    _poison(cache)
    for what, steps in (("whole", trace_whole(reqs)), ("pieces", trace_chunks(reqs, pieces=(70, 1, 33))),
                        ("batch", trace_batches([{"a": (reqs["a"], 20), "b": (reqs["b"], 8)}]))):
        _check(replay(model, cache, steps), cfg, w, reqs, plain, dtype, f"wider model, {what}, {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point_and_the_replay_program(folders, cuda_device, tmp_path, dtype):
    cfg = rc.CASE_A
    d, w = folders["A", dtype]
    V = cfg["vocab"]
    model = bn.load_model(d, dtype=dtype)
    prompts = [random_tokens(31, 50, V), random_tokens(32, 3, V), random_tokens(33, 120, V)]
    got = bn.generate(model, prompts, max_new_tokens=[70, 20, 24])
    for p, g in zip(prompts, got):
        assert len(g.tokens) in (70, 20, 24) and g.finish_reason == "length"
        seq = list(p) + g.tokens[:-1]
        ref = pr.forward(seq, w, cfg)[len(p) - 1:]
        if dtype == "float32":
            slack = 2 * TOL_F32 * max(1.0, float(np.abs(ref).max()))
        else:
            slack = 2 * BF16_GAP_FACTOR * float(np.abs(pr.forward(seq, w, cfg, r=pr.to_bf16)[len(p) - 1:] - ref).max())
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
    plain = {k: pr.forward(t, w, cfg) for k, t in reqs.items()}
    _check(collect_trace_output(steps, out, V), cfg, w, reqs, plain, dtype, "through bin/trace_run")


def test_the_command_line_writes_a_random_model_of_the_design_and_generates_from_it(tmp_path, cuda_device):
    cfgp = tmp_path / "cfg.json"
    cfgp.write_text(json.dumps(rc.CASE_C))
    folder = tmp_path / "m"
    cmd = [sys.executable, os.path.join(ROOT, "bin", "bitnet"), str(folder), "--random-weights", "--config", str(cfgp),
           "--weight-seed", "3", "--dtype", "float32", "--prompt-token-ids", "5,17,3,9,9,1", "--prompt-token-ids", "7",
           "-n", "9", "--repeat-penalty", "1.0", "--token-ids"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    lines = [[int(t) for t in l.split(",")] for l in p.stdout.splitlines() if l.strip()]
    assert [len(l) for l in lines] == [9, 9] and "Generation complete tokens=18" in p.stderr

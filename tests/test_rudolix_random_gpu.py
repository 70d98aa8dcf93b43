"""Rudolix configurations drawn at random by fixed seeds from all that its config.json allows (numbers of layers and their
kinds in any order, streams, taps, head counts and sizes with key and value widths apart, groups, parts of the output
norm, rotated parts of any even width, experts of which a token takes one, some or all, layers without a
feed-forward), each stepped whole, token by token, in pieces and in unequal batches against the plain statement, in both
number formats."""
import numpy as np
import pytest

import bitnet_c_b200 as bn
import plain_rudolix as pr
import rudolix_cases as rc
from helpers import TOL_F32, random_tokens, replay, trace_batches, trace_chunks, trace_tail, trace_whole
from test_rudolix_gpu import _poison, _plain_rounded

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", autouse=True)
def _give_device_memory_back():
    """The models and caches of this module leave the allocator's pool when it is done."""
    yield
    import gc
    import torch as _torch
    gc.collect()
    if _torch.cuda.is_available():
        _torch.cuda.empty_cache()


def draw_config(seed: int):
    rng = np.random.default_rng(seed)
    pick = lambda xs: xs[int(rng.integers(len(xs)))]
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        kind = pick(["attention", "delta", "mamba2"])
        g = pick([1, 2, 3, 4])
        heads = g * pick([1, 2, 3, 4])
        if kind == "attention":
            dim = pick([4, 8, 16, 20, 32, 64])
            m = {"heads": heads, "kv_heads": g, "dim": dim, "vdim": pick([4, 8, 12, 16, 32, 48]), "scale": float(rng.uniform(0.15, 0.8)),
                 "rot": {"base": float(pick([100.0, 1e4, 1e6])), "dims": 2 * int(rng.integers(1, dim // 2 + 1))}}
        elif kind == "delta":
            m = {"heads": heads, "kv_heads": g, "dim": pick([4, 6, 8, 16, 32, 40, 64, 96]), "vdim": pick([4, 5, 8, 16, 32, 48, 72]),
                 "conv": int(rng.integers(1, 7))}
        else:
            vdim = pick([4, 5, 8, 16, 32, 48, 72])
            parts = [p for p in range(1, heads * vdim + 1) if heads * vdim % p == 0 and heads * vdim // p >= 4]
            m = {"heads": heads, "groups": g, "state": pick([4, 6, 8, 16, 32, 40, 64, 96]), "vdim": vdim, "conv": int(rng.integers(1, 7)),
                 "norm_groups": pick(parts)}
        mlp = None
        if rng.random() < 0.8:
            e = pick([1, 2, 3, 5, 8, 16])
            mlp = pick([{"kind": "dense", "ff": pick([8, 12, 37, 64, 130])},
                        {"kind": "moe", "router": {"experts": e, "top": int(rng.integers(1, min(e, 4) + 1))},
                         "expert": {"ff": pick([8, 12, 24, 40]), "limit": float(pick([0.5, 1.0, 3.0, 7.0]))}}])
        layers.append({"type": kind, "mixer": m, "mlp": mlp})
    return {"architecture": "Rudolix", "vocab": int(rng.integers(50, 300)), "width": pick([32, 40, 48, 50, 64, 72, 96, 128]),
            "streams": int(rng.integers(1, 7)), "residual_mult": float(pick([0.25, 0.5, 1.0])), "norm": {"eps": pick([1e-5, 1e-6])},
            "canon": {"taps": int(rng.integers(1, 7))}, "embedding": {"scale": float(pick([1.0, 4.0, 16.0]))}, "layers": layers}


@pytest.mark.parametrize("seed", range(14))
def test_a_configuration_drawn_at_random_steps_like_the_plain_statement(tmp_path, cuda_device, seed):
    cfg = draw_config(7000 + seed)
    V = cfg["vocab"]
    reqs = {"a": random_tokens(seed, 230, V), "b": random_tokens(seed + 50, 1, V), "c": random_tokens(seed + 99, 70, V)}
    for dtype in ("float32", "bfloat16") if seed % 2 == 0 else ("float32",):
        # with routers whose choices hang on more than rounding
        w = rc.draw_weights(cfg, seed=seed, calm=True)
        plain = {r: pr.forward(t, w, cfg) for r, t in reqs.items()}
        # how much single-precision rounding may move a position shows when the plain statement runs with weights
        # moved by 1e-7 of their size; float32 is allowed 30 times that on top of its bound
        rng = np.random.default_rng(seed)
        moved = {k: a * (1.0 + 1e-7 * rng.standard_normal(a.shape)) for k, a in w.items()}
        slack = {r: 30.0 * np.abs(pr.forward(t, moved, cfg) - plain[r]).max(axis=1) for r, t in reqs.items()}
        model = bn.load_model(rc.write_folder(str(tmp_path / dtype), cfg, w), dtype=dtype)
        cache = model.new_cache(max_tokens=64 * 10, max_seqs=3)
        _poison(cache)
        for what, steps in (("whole", trace_whole(reqs)), ("last 25 one by one", trace_tail(reqs, 25)),
                            ("pieces", trace_chunks(reqs, pieces=(3, 64, 17, 1))),
                            ("an unequal batch", trace_batches([{"a": (reqs["a"], 12), "c": (reqs["c"], 30), "b": (reqs["b"], 0)}]))):
            got = replay(model, cache, steps)
            for r, per_pos in got.items():
                assert all(np.isfinite(row).all() for row in per_pos.values()), f"seed {seed}: {what}: request {r}"
                err = np.array([np.abs(row.astype(np.float64) - plain[r][p]).max() for p, row in sorted(per_pos.items())])
                places = sorted(per_pos)
                if dtype == "bfloat16":
                    # a model drawn at random may be rough: the bound follows what rounding the stored activations does
                    # to the plain statement (three times the request's largest gap, a fifth of the positions beyond
                    # three times its 80th percentile)
                    gap = np.abs(plain[r] - _plain_rounded(cfg, w, reqs[r])).max(axis=1)[places]
                    assert err.max() <= 3.0 * gap.max() + 1e-3, f"seed {seed}: {what}, {dtype}: request {r}: position {places[int(err.argmax())]}"
                    assert int((err > 3.0 * np.percentile(gap, 80) + 1e-3).sum()) <= max(1, len(err) // 5), f"seed {seed}: {what}, {dtype}: request {r}"
                    continue
                bound = TOL_F32 * max(1.0, float(np.abs(plain[r]).max())) + slack[r][places]
                assert (err <= bound).all(), f"seed {seed}: {what}: request {r} position {places[int((err - bound).argmax())]}: {err.max():.3e}"
        model.check_kernels()

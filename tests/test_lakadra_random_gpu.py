"""Lakadra configurations drawn at random by fixed seeds from all that its config.json allows (numbers of layers and their
kinds in any order, readers of any earlier latent layer, head counts and sizes with key and value widths apart, windows,
rotated parts, factors of both signs, taps and blocks, experts and identity experts in groups, layers without a
feed-forward), each stepped whole, token by token, in pieces and in unequal batches against the plain statement, in both
number formats."""
import numpy as np
import pytest

import bitnet_c_b200 as bn
import lakadra_cases as lc
import plain_lakadra as pl
from helpers import TOL_F32, random_tokens, replay, trace_batches, trace_chunks, trace_tail, trace_whole
from test_lakadra_gpu import _plain_rounded, _poison

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
    layers, sources = [], []
    for i in range(int(rng.integers(1, 6))):
        kind = pick(["lightning", "latent_attention", "parallel"])
        if kind == "lightning":
            heads = pick([1, 2, 3, 4, 6])
            m = {"heads": heads, "dim": pick([4, 6, 8, 16, 32, 40, 64, 96]), "vdim": pick([4, 5, 8, 16, 32, 48, 72]),
                 "decay": [float(d) for d in 1 - 10.0 ** -rng.uniform(0, 4, heads)]}
        elif kind == "latent_attention":
            heads, dim, vdim, q = pick([1, 2, 3, 4, 8]), pick([4, 8, 16, 20, 32, 64]), pick([4, 8, 12, 16, 32, 48]), pick([5, 8, 24, 40])
            scale = float(rng.uniform(0.15, 0.8))
            if sources and rng.random() < 0.5:
                j = pick(sources)
                src = layers[j]["mixer"]
                m = lc.latent(heads, dim, src["rot_dim"], vdim, q, src["kv_rank"], scale, src["rot"]["base"], kv_from=j)
            else:
                sources.append(i)
                m = lc.latent(heads, dim, pick([2, 4, 8, 16, 32]), vdim, q, pick([8, 12, 24, 48, 96, 240, 288]), scale, float(pick([100.0, 1e4, 1e6])))
        else:
            g = pick([1, 2, 3, 4])
            dim, blocks = pick([4, 8, 16, 20, 32, 64]), pick([1, 2, 3, 5])
            m = lc.pair(g * pick([1, 2, 3, 4]), g, dim, pick([4, 8, 12, 16, 32, 48]), pick([1, 2, 17, 40, 64, 65, 128, 500]),
                        2 * int(rng.integers(1, dim // 2 + 1)), float(pick([100.0, 1e4, 1e6])), pick([None, 0.5, 2.0, 8.0]),
                        float(rng.uniform(0.15, 0.8)), blocks * pick([4, 7, 16, 24]), blocks, int(rng.integers(1, 7)),
                        float(rng.uniform(-1.5, 1.5)), float(rng.uniform(-1.5, 1.5)))
        mlp = None
        if rng.random() < 0.8:
            groups, size = pick([1, 2, 3, 4]), pick([1, 2, 3, 5])
            n = groups * size
            identity, keep = int(rng.integers(0, n)), int(rng.integers(1, groups + 1))
            mlp = lc.moe(n - identity, identity, int(rng.integers(1, min(keep * size, 4) + 1)), groups, keep, pick([8, 12, 24, 40]), pick([8, 13, 40]))
        layers.append({"type": kind, "mixer": m, "mlp": mlp})
    return {"architecture": "Lakadra", "vocab": int(rng.integers(50, 300)), "width": pick([32, 40, 48, 50, 64, 72, 96, 128]), "norm": {"eps": pick([1e-5, 1e-6])},
            "logit_scale": float(rng.uniform(0.3, 1.5)), "logit_softcap": float(pick([5.0, 15.0, 30.0])), "layers": layers}


@pytest.mark.parametrize("seed", range(16))
def test_a_configuration_drawn_at_random_steps_like_the_plain_statement(tmp_path, cuda_device, seed):
    cfg = draw_config(8000 + seed)
    V = cfg["vocab"]
    reqs = {"a": random_tokens(seed, 230, V), "b": random_tokens(seed + 50, 1, V), "c": random_tokens(seed + 99, 70, V)}
    for dtype in ("float32", "bfloat16") if seed % 2 == 0 else ("float32",):
        w = lc.draw_weights(cfg, seed=seed, calm=True)  # with routers whose choices hang on more than rounding
        plain = {r: pl.forward(t, w, cfg) for r, t in reqs.items()}
        # how much single-precision rounding may move a position shows when the plain statement runs with weights
        # moved by 1e-7 of their size; float32 is allowed 30 times that on top of its bound
        rng = np.random.default_rng(seed)
        moved = {k: a * (1.0 + 1e-7 * rng.standard_normal(a.shape)) for k, a in w.items()}
        slack = {r: 30.0 * np.abs(pl.forward(t, moved, cfg) - plain[r]).max(axis=1) for r, t in reqs.items()}
        model = bn.load_model(lc.write_folder(str(tmp_path / dtype), cfg, w), dtype=dtype)
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

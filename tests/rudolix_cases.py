"""Small Rudolix configurations and weights for the tests.

The weights are drawn here, by tensor name and shape as the design names them (not from the library's parameter
table), with scales that make faults show: queries and keys with scores that spread over several units; sinks around
three, so that a softmax without them is visibly another; decays from a few tokens to thousands, so that a state that is
lost or cut shows far on; streams that are read, mixed and written with numbers far from each other; gains, biases and
layer scales well away from one and zero; router biases of the size of the logits (``calm``: biases a unit apart and products
well below that, so that an activation's rounding hardly ever changes a choice; otherwise a choice hangs on every
token, and only single precision can be held to it).  All values are exactly
representable in bfloat16, so the same folder serves both number formats.
"""
import json
import os

import numpy as np
import torch

from plain_rudolix import to_bf16

# every size differs from layer to layer; three streams; heads that share queries and keys, or the state's input and
# read-out, two or three at a time; value widths apart from key widths; a rotated part narrower than the head; a
# layer without a feed-forward; experts of which a token takes some, all, or the only one
CASE_A = {
    "architecture": "Rudolix", "vocab": 97, "width": 64, "streams": 3, "residual_mult": 0.7, "norm": {"eps": 1e-5},
    "canon": {"taps": 4}, "embedding": {"scale": 3.0},
    "layers": [
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.4, "rot": {"base": 1000.0, "dims": 8}},
         "mlp": {"kind": "moe", "router": {"experts": 5, "top": 2}, "expert": {"ff": 24, "limit": 1.5}}},
        {"type": "delta", "mixer": {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 20, "conv": 3}, "mlp": {"kind": "dense", "ff": 56}},
        {"type": "mamba2", "mixer": {"heads": 4, "groups": 2, "state": 24, "vdim": 12, "conv": 5, "norm_groups": 2}, "mlp": None},
        {"type": "mamba2", "mixer": {"heads": 3, "groups": 1, "state": 8, "vdim": 40, "conv": 2, "norm_groups": 3},
         "mlp": {"kind": "moe", "router": {"experts": 3, "top": 3}, "expert": {"ff": 16, "limit": 0.8}}},
        {"type": "delta", "mixer": {"heads": 2, "kv_heads": 2, "dim": 32, "vdim": 8, "conv": 4},
         "mlp": {"kind": "moe", "router": {"experts": 1, "top": 1}, "expert": {"ff": 40, "limit": 2.5}}},
    ],
}

# sizes that are no multiples of 8 (and mostly not of 4) anywhere: rows of no whole 16-byte pieces, so the kernels take
# their number-by-number paths and the recurrences go token by token; one stream; convolutions of one tap; one
# key/value head
CASE_B = {
    "architecture": "Rudolix", "vocab": 61, "width": 50, "streams": 1, "residual_mult": 1.0, "norm": {"eps": 1e-6},
    "canon": {"taps": 2}, "embedding": {"scale": 1.0},
    "layers": [
        {"type": "delta", "mixer": {"heads": 3, "kv_heads": 1, "dim": 10, "vdim": 7, "conv": 1}, "mlp": {"kind": "dense", "ff": 37}},
        {"type": "mamba2", "mixer": {"heads": 5, "groups": 5, "state": 6, "vdim": 9, "conv": 3, "norm_groups": 5},
         "mlp": {"kind": "moe", "router": {"experts": 4, "top": 1}, "expert": {"ff": 18, "limit": 1.0}}},
        {"type": "attention", "mixer": {"heads": 3, "kv_heads": 1, "dim": 10, "vdim": 7, "scale": 0.5, "rot": {"base": 77.0, "dims": 10}},
         "mlp": None},
    ],
}

# key and value rows in multiples of 16 (the tensor-core kernel for runs of tokens); a whole head rotated; heads of the
# delta rule all on one query/key head; four streams; state-space heads of 64 x 32 numbers in two groups
CASE_C = {
    "architecture": "Rudolix", "vocab": 150, "width": 96, "streams": 4, "residual_mult": 0.4, "norm": {"eps": 1e-6},
    "canon": {"taps": 3}, "embedding": {"scale": 2.0},
    "layers": [
        {"type": "mamba2", "mixer": {"heads": 4, "groups": 2, "state": 64, "vdim": 32, "conv": 4, "norm_groups": 1},
         "mlp": {"kind": "moe", "router": {"experts": 6, "top": 3}, "expert": {"ff": 32, "limit": 1.2}}},
        {"type": "attention", "mixer": {"heads": 8, "kv_heads": 4, "dim": 32, "vdim": 16, "scale": 0.3, "rot": {"base": 50000.0, "dims": 32}},
         "mlp": {"kind": "dense", "ff": 200}},
        {"type": "delta", "mixer": {"heads": 4, "kv_heads": 1, "dim": 64, "vdim": 48, "conv": 4},
         "mlp": {"kind": "moe", "router": {"experts": 4, "top": 2}, "expert": {"ff": 48, "limit": 3.0}}},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 4, "dim": 16, "vdim": 64, "scale": 0.6, "rot": {"base": 300.0, "dims": 12}},
         "mlp": {"kind": "dense", "ff": 72}},
    ],
}

CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C}


def layer_shapes(cfg: dict, i: int) -> dict:
    """The tensors of one layer by name."""
    layer, W, S, p = cfg["layers"][i], cfg["width"], cfg["streams"], f"l{i}."
    m, kind = layer["mixer"], layer["type"]
    t = {}
    if kind == "attention":
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        t.update({"q": (H * d, W), "k": (G * d, W), "v": (G * dv, W), "sink": (H,), "o": (W, H * dv)})
    elif kind == "delta":
        H, G, d, dv, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        t.update({"q": (G * d, W), "q.conv": (G * d, n), "k": (G * d, W), "k.conv": (G * d, n), "v": (H * dv, W), "v.conv": (H * dv, n),
                  "b": (H, W), "a": (H, W), "A_log": (H,), "dt_bias": (H,), "norm": (dv,), "g": (H * dv, W), "o": (W, H * dv)})
    else:
        H, G, N, P, n = m["heads"], m["groups"], m["state"], m["vdim"], m["conv"]
        ch = H * P + 2 * G * N
        t.update({"in": (H * P + ch + H, W), "conv": (ch, n), "conv.b": (ch,), "dt_bias": (H,), "A_log": (H,), "D": (H,),
                  "norm": (H * P,), "o": (W, H * P)})
    t = {p + "mix." + k: v for k, v in t.items()}
    mlp = layer.get("mlp")
    for q in (1, 2) if mlp is not None else (1,):
        t.update({p + f"norm{q}": (W,), p + f"norm{q}.b": (W,), p + f"ls{q}": (W,), p + f"hc{q}.in": (S,), p + f"hc{q}.out": (S,),
                  p + f"hc{q}.mix": (S, S), p + f"canon{q}": (W, cfg["canon"]["taps"])})
    if mlp is not None and mlp["kind"] == "dense":
        t.update({p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"]), p + "mlp.act": (4,)})
    elif mlp is not None:
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        t.update({p + "mlp.router": (E, W), p + "mlp.router.b": (E,)})
        for e in range(E):
            t.update({p + f"mlp.e{e}.gate": (ff, W), p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
    return t


def tensor_shapes(cfg: dict) -> dict:
    """Every tensor of the design by name, from the configuration."""
    W = cfg["width"]
    t = {"embed": (cfg["vocab"], W), "final.norm": (W,), "final.norm.b": (W,)}
    for i in range(len(cfg["layers"])):
        t.update(layer_shapes(cfg, i))
    return t


def draw_weights(cfg: dict, seed: int, calm: bool = False) -> dict:
    rng = np.random.default_rng(seed)
    S = cfg["streams"]
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = rng.standard_normal(shape)
        last = name.split(".")[-1]
        if name.endswith((".norm", "norm1", "norm2")):
            a = 1.0 + 0.3 * z
        elif name.endswith(("norm.b", "norm1.b", "norm2.b")):
            a = 0.2 * z
        elif last == "embed":
            a = z
        elif last in ("ls1", "ls2"):
            a = 0.8 + 0.3 * z
        elif last == "in" and ".hc" in name:
            a = (1.0 + 0.4 * z) / np.sqrt(S) * np.where(np.arange(S) % 2, -0.6, 1.0)  # the streams are not simply added up
        elif last == "out":
            a = 1.0 + 0.3 * z
        elif last == "mix":
            a = 0.75 * np.eye(S) + 0.3 * z / np.sqrt(S)
        elif last in ("canon1", "canon2"):
            a = 0.3 * z
        elif last == "conv":
            a = 0.6 * z
        elif name.endswith("conv.b"):
            a = 0.3 * z
        elif last == "sink":
            a = z + 3.0
        elif last == "A_log":
            a = rng.uniform(-4.0, 0.5, shape)
        elif last == "dt_bias":
            a = rng.uniform(-4.0, -0.5, shape)
        elif last == "D":
            a = 0.8 + 0.3 * z
        elif last == "act":
            a = np.array([0.7, 0.45, 0.5, 0.35]) * (1.0 + 0.2 * z)
        elif name.endswith("router.b"):
            a = rng.permutation(shape[0]) - 0.5 * (shape[0] - 1) if calm else 0.7 * z
        elif last == "router":
            a = z * (0.3 if calm else 1.2) / np.sqrt(shape[-1])
        elif last in ("o", "down"):
            a = z * 0.7 / np.sqrt(shape[-1])
        else:
            a = z * 1.2 / np.sqrt(shape[-1])
        out[name] = to_bf16(np.asarray(a, dtype=np.float64))
    return out


def write_folder(folder: str, cfg: dict, weights: dict, storage: str = "bfloat16") -> str:
    from bitnet_c_b200.weights import write_safetensors
    os.makedirs(folder, exist_ok=True)
    dt = {"bfloat16": torch.bfloat16, "float32": torch.float32}[storage]
    write_safetensors(os.path.join(folder, "model.safetensors"),
                      [(n, torch.tensor(np.asarray(a, dtype=np.float32)).to(dt)) for n, a in weights.items()])
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    return folder

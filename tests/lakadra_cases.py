"""Small Lakadra configurations and weights for the tests.

The weights are drawn here, by tensor name and shape as the design names them (not from the library's parameter table),
with scales that make faults show: queries and keys with scores that spread over several units; decays from a few tokens to
thousands, so that a state that is lost or cut shows far on; biases and gains well away from zero and one; corrections that
change the router's choice and are mostly negative, so that an expert of a group that is left out would win if it counted as
zero (``calm``: corrections far apart and router products well below that, so that an activation's rounding hardly ever
changes a choice; otherwise a choice hangs on every token, and only single precision can be held to it).  All values are
exactly representable in bfloat16, so the same folder serves both number formats.
"""
import json
import os

import numpy as np
import torch

from plain_lakadra import to_bf16


def moe(experts, identity, top, groups, keep, ff, shared):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}},
            "expert": {"ff": ff}, "shared": {"ff": shared}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, **more):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim}, **more}


def pair(heads, kv_heads, dim, vdim, window, dims, base, factor, scale, width, blocks, conv, left_scale=0.8, right_scale=1.1):
    rot = {"base": base, "dims": dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    return {"left_scale": left_scale, "right_scale": right_scale,
            "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}, "rot": rot},
            "right": {"width": width, "blocks": blocks, "conv": conv}}


# every size differs from layer to layer; two sources of latents and a reader of each; heads that share keys two or three at a
# time; windows shorter and longer than a page; a layer without a feed-forward; rows in multiples of 16 in one place and of
# nothing in the next
CASE_A = {
    "architecture": "Lakadra", "vocab": 97, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 0.7, "logit_softcap": 12.0,
    "layers": [
        {"type": "latent_attention", "mixer": latent(3, 16, 8, 20, 40, 24, 0.5, 300.0), "mlp": moe(5, 1, 2, 3, 2, 24, 40)},
        {"type": "parallel", "mixer": pair(6, 2, 16, 24, 37, 8, 1000.0, 3.0, 0.4, 48, 4, 3), "mlp": moe(4, 4, 3, 2, 1, 16, 24)},
        {"type": "lightning", "mixer": {"heads": 3, "dim": 12, "vdim": 20, "decay": [0.7, 0.97, 0.9995]}, "mlp": None},
        {"type": "latent_attention", "mixer": latent(5, 8, 8, 12, 24, 24, 0.7, 300.0, kv_from=0), "mlp": moe(6, 2, 2, 4, 3, 40, 16)},
        {"type": "latent_attention", "mixer": latent(2, 32, 16, 48, 32, 48, 0.3, 5000.0), "mlp": moe(3, 0, 3, 1, 1, 16, 8)},
        {"type": "parallel", "mixer": pair(4, 4, 32, 16, 100, 32, 50000.0, None, 0.3, 96, 3, 5, -0.6, 0.5), "mlp": moe(7, 2, 1, 9, 4, 32, 48)},
        {"type": "lightning", "mixer": {"heads": 4, "dim": 32, "vdim": 16, "decay": [0.5, 0.9, 0.99, 0.999]}, "mlp": moe(2, 2, 2, 2, 2, 48, 32)},
        {"type": "latent_attention", "mixer": latent(4, 16, 16, 16, 16, 48, 0.5, 5000.0, kv_from=4), "mlp": None},
    ],
}

# sizes that are no multiples of 8 (and mostly not of 4) anywhere: rows of no whole 16-byte pieces, so the kernels take
# their number-by-number paths and the lightning state goes token by token; no soft cap; one tap; a window of one token
CASE_B = {
    "architecture": "Lakadra", "vocab": 61, "width": 50, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "logit_softcap": 30.0,
    "layers": [
        {"type": "parallel", "mixer": pair(3, 1, 10, 7, 1, 6, 77.0, 1.0, 0.5, 35, 5, 1), "mlp": moe(4, 1, 2, 5, 3, 18, 11)},
        {"type": "lightning", "mixer": {"heads": 3, "dim": 10, "vdim": 7, "decay": [0.3, 0.99, 0.95]}, "mlp": moe(5, 1, 1, 1, 1, 13, 37)},
        {"type": "latent_attention", "mixer": latent(3, 9, 6, 7, 13, 19, 0.6, 1000.0), "mlp": None},
        {"type": "parallel", "mixer": pair(2, 2, 6, 9, 65, 2, 10.0, 8.0, 0.7, 22, 2, 4), "mlp": moe(1, 0, 1, 1, 1, 9, 5)},
        {"type": "latent_attention", "mixer": latent(1, 11, 6, 5, 7, 19, 0.9, 1000.0, kv_from=2), "mlp": moe(3, 3, 2, 3, 2, 10, 6)},
    ],
}

# heads of 64 and 128, key rows of more than 256 numbers (keys and values made per head in prompts), windows at a page's edge
CASE_C = {
    "architecture": "Lakadra", "vocab": 150, "width": 128, "norm": {"eps": 1e-6}, "logit_scale": 0.5, "logit_softcap": 20.0,
    "layers": [
        {"type": "latent_attention", "mixer": latent(4, 64, 32, 64, 64, 256, 0.2, 1e5), "mlp": moe(6, 2, 3, 4, 2, 64, 96)},
        {"type": "lightning", "mixer": {"heads": 2, "dim": 64, "vdim": 128, "decay": [0.98, 0.9999]}, "mlp": moe(8, 0, 2, 2, 1, 32, 64)},
        {"type": "parallel", "mixer": pair(4, 1, 128, 64, 64, 64, 1e4, 4.0, 0.1, 256, 2, 4), "mlp": moe(4, 4, 2, 4, 3, 48, 64)},
        {"type": "latent_attention", "mixer": latent(2, 128, 32, 128, 48, 256, 0.15, 1e5, kv_from=0), "mlp": moe(6, 2, 2, 2, 2, 64, 32)},
    ],
}

CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C}


def layer_shapes(cfg: dict, i: int) -> dict:
    """The tensors of one layer by name."""
    layer, W, p = cfg["layers"][i], cfg["width"], f"l{i}."
    m, kind = layer["mixer"], layer["type"]
    if kind == "lightning":
        qk, vv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        t = {"q": (qk, W), "k": (qk, W), "v": (vv, W), "g": (vv, W), "norm": (vv,), "o": (W, vv)}
    elif kind == "latent_attention":
        H, c = m["heads"], m["kv_rank"]
        t = {"dq": (m["q_rank"], W), "dq.norm": (m["q_rank"],), "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
             "uk": (H * m["dim"], c), "uv": (H * m["vdim"], c), "o": (W, H * m["vdim"])}
        if m.get("kv_from") is None:
            t.update({"dkv": (c + m["rot_dim"], W), "dkv.norm": (c,)})
    else:
        a, b = m["left"], m["right"]
        H, G, d, dv, n, B = a["heads"], a["kv_heads"], a["dim"], a["vdim"], b["width"], b["blocks"]
        t = {"left.q": (H * d, W), "left.q.b": (H * d,), "left.k": (G * d, W), "left.k.b": (G * d,), "left.v": (G * dv, W), "left.v.b": (G * dv,),
             "left.g": (H, W), "left.o": (W, H * dv), "left.o.b": (W,), "right.y": (n, W), "right.y.b": (n,), "right.x": (n, W), "right.x.b": (n,),
             "right.conv": (n, b["conv"]), "right.conv.b": (n,), "right.ra": (B, n // B, n // B), "right.ra.b": (B, n // B),
             "right.ri": (B, n // B, n // B), "right.ri.b": (B, n // B), "right.lam": (n,), "right.o": (W, n)}
    t = {p + "mix." + k: v for k, v in t.items()}
    t[p + "norm1"] = (W,)
    mlp = layer.get("mlp")
    if mlp:
        ro, ff = mlp["router"], mlp["expert"]["ff"]
        n = ro["experts"] + ro.get("identity", 0)
        t.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
        for e in range(ro["experts"]):
            t.update({p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
        if mlp.get("shared"):
            s = mlp["shared"]["ff"]
            t.update({p + "mlp.shared.up": (s, W), p + "mlp.shared.down": (W, s), p + "mlp.shared.sg": (1, W)})
    return t


def tensor_shapes(cfg: dict) -> dict:
    """Every tensor of the design by name, from the configuration."""
    W = cfg["width"]
    t = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    for i in range(len(cfg["layers"])):
        t.update(layer_shapes(cfg, i))
    return t


def draw_weights(cfg: dict, seed: int, calm: bool = False) -> dict:
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = rng.standard_normal(shape)
        last = name.split(".")[-1]
        if last == "norm1" or name == "final.norm":
            a = 0.3 * z  # gains stored as their distance from one
        elif last == "norm":
            a = 1.0 + 0.3 * z
        elif last == "embed":
            a = z
        elif last == "head":
            a = z * 3.0 / np.sqrt(shape[-1])
        elif last == "correction":
            a = 0.7 * (rng.permutation(shape[0]) - shape[0]) if calm else 0.25 * z - 0.6
        elif last == "router":
            a = z * (0.3 if calm else 1.2) / np.sqrt(shape[-1])
        elif last == "lam":
            a = rng.uniform(-7.0, -1.5, shape)
        elif last == "conv":
            a = 0.6 * z
        elif last == "b":
            a = 0.4 * z
        elif last == "sg":
            a = 2.0 * z / np.sqrt(shape[-1])
        elif last in ("o", "down"):
            a = z * 0.8 / np.sqrt(shape[-1])
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

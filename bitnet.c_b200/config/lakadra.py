"""Lakadra: a decoder of parallel blocks whose layers are listed one by one in ``config.json``.

Every layer norms the stream once (the gain stored as its distance from one); a mixer and a mixture of experts both read
that norm, and the sum of their results is added.  The mixer is linear attention under one fixed decay per head
(``lightning``), softmax attention through low-rank latents that a later layer may share (``latent_attention``), or a pair
(``parallel``): grouped-query attention over a sliding window with biases, slowed-down rotary positions, one added to the
softmax's denominator and a gate per head, beside a real-gated linear recurrence behind a short convolution, each with a
factor.  The experts are ungated squared-relu units, chosen within the best groups of experts by softmax scores plus a
correction; some of the router's outputs stand for the input itself, and a shared expert with a gate of its own runs for
every token.  The keys of ``config.json``:

    architecture            "Lakadra"
    vocab, width            sizes of the embedding and the residual stream
    norm.eps                eps of every norm
    logit_scale             factor on the head's product
    logit_softcap           (optional) c: logits become c tanh(logits / c)
    layers[i].type          "lightning" | "latent_attention" | "parallel"
    layers[i].mixer         lightning: heads, dim, vdim, decay (one number per head);
                            latent_attention: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot.base, rot.dims,
                            kv_from (optional: the layer whose cached rows this one reads);
                            parallel: left_scale, right_scale; left: heads, kv_heads, dim, vdim, scale, mask.size, rot.base,
                            rot.dims, rot.scaling.factor (optional); right: width, blocks, conv
    layers[i].mlp           null, or kind "moe" with router.experts, router.top, router.identity (optional),
                            router.groups (optional: count, keep), expert.ff, shared (optional: ff)
    max_positions           (optional) the longest sequence; the design itself has no limit
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Any, Dict, List

from .spec import (BiasAttentionSpec, ConfigError, GatedLinearSpec, LatentAttentionSpec, LightningSpec, LinearHeadSpec,
                   ModelSpec, MoeSpec, PairSpec, ParallelBlockSpec, RmsNormSpec, RotaryBlendSpec, ScheduleEntry)

ARCHITECTURE = "Lakadra"
DEFAULT_MAX_POSITIONS = 1 << 20


def _need(d: Dict[str, Any], key: str, where: str) -> Any:
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: {where} has no '{key}'")
    return d[key]


def _int(d, key, where, minimum=1, maximum=None) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v < minimum or (maximum is not None and v > maximum):
        upto = f" and at most {maximum}" if maximum is not None else ""
        raise ConfigError(f"config.json: {where}.{key} must be an integer of at least {minimum}{upto}, got {v!r}")
    return v


def _num(d, key, where) -> float:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
    return float(v)


def _positive(d, key, where) -> float:
    v = _num(d, key, where)
    if not v > 0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v!r}")
    return v


def _multiple(m: Dict[str, Any], key: str, of: str, where: str) -> int:
    """m[key], which must be a multiple of m[of]."""
    a, b = _int(m, key, where), _int(m, of, where)
    if a % b:
        raise ConfigError(f"config.json: {where}: {key}={a} is not a multiple of {of}={b}")
    return a


def _rotary(m: Dict[str, Any], where: str, most: int, pairing: str) -> RotaryBlendSpec:
    rot, at = _need(m, "rot", where), where + ".rot"
    dims = _int(rot, "dims", at, minimum=2, maximum=min(most, 512))
    if dims % 2:
        raise ConfigError(f"config.json: {at}.dims={dims} must be even")
    scaling = rot.get("scaling")
    slowdown = 1.0 if scaling is None else _positive(scaling, "factor", at + ".scaling")
    return RotaryBlendSpec(dims=dims, base=_positive(rot, "base", at), pairing=pairing, slowdown=slowdown)


@dataclass(frozen=True)
class LakadraConfig:
    """The file as it was read (``text``: canonical JSON, so that the record is hashable and can be written back
    unchanged) plus the checked top-level numbers."""

    text: str
    vocab: int
    width: int
    n_layers: int
    max_positions: int

    @property
    def data(self) -> Dict[str, Any]:
        return json.loads(self.text)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "LakadraConfig":
        layers = _need(d, "layers", "the file")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        mp = d.get("max_positions") or DEFAULT_MAX_POSITIONS
        cfg = cls(text=json.dumps(d, sort_keys=True), vocab=_int(d, "vocab", "the file"), width=_int(d, "width", "the file"),
                  n_layers=len(layers), max_positions=int(mp))
        cfg.to_spec()  # every layer is checked by building its spec
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return self.data

    def with_max_positions(self, max_seq: int) -> "LakadraConfig":
        if max_seq and 0 < max_seq < self.max_positions:
            d = self.data
            d["max_positions"] = int(max_seq)
            return LakadraConfig.from_dict(d)
        return self

    # ---- translation into parts ------------------------------------------------------------
    def _lightning(self, m: Dict[str, Any], where: str, eps: float) -> LightningSpec:
        heads, decay = _int(m, "heads", where), _need(m, "decay", where)
        if not isinstance(decay, list) or len(decay) != heads or not all(
                isinstance(v, (int, float)) and not isinstance(v, bool) and 0 <= v <= 1 for v in decay):
            raise ConfigError(f"config.json: {where}.decay must list one number from 0 to 1 for each of the {heads} heads, got {decay!r}")
        return LightningSpec(width=self.width, n_heads=heads, head_dim=_int(m, "dim", where, maximum=256),
                             v_head_dim=_int(m, "vdim", where), decay=tuple(float(v) for v in decay), norm_eps=eps)

    def _latent(self, i: int, layers: List[Any], m: Dict[str, Any], where: str, eps: float) -> LatentAttentionSpec:
        rot_dim = _int(m, "rot_dim", where, minimum=2)
        position = _rotary(m, where, rot_dim, "neighbours")
        if position.dims != rot_dim:
            raise ConfigError(f"config.json: {where}: rot.dims={position.dims} must equal rot_dim={rot_dim}")
        spec = LatentAttentionSpec(
            width=self.width, n_heads=_int(m, "heads", where), head_dim=_int(m, "dim", where), rot_dim=rot_dim,
            v_head_dim=_int(m, "vdim", where), q_rank=_int(m, "q_rank", where), kv_rank=_int(m, "kv_rank", where),
            scale=_num(m, "scale", where), position=position, norm_eps=eps, head_gate=False, own_kv=m.get("kv_from") is None)
        if spec.kv_rank + rot_dim > 2048:
            raise ConfigError(f"config.json: {where}: kv_rank + rot_dim = {spec.kv_rank + rot_dim} must be at most 2048")
        if not spec.own_kv:
            j = _int(m, "kv_from", where, minimum=0, maximum=max(i - 1, 0))
            source = layers[j] if j < i and isinstance(layers[j], dict) else {}
            src = source.get("mixer") or {}
            if source.get("type") != "latent_attention" or src.get("kv_from") is not None:
                raise ConfigError(f"config.json: {where}.kv_from={j} names no earlier latent_attention layer with rows of its own")
            if any(src.get(k) != m.get(k) for k in ("kv_rank", "rot_dim", "rot")):
                raise ConfigError(f"config.json: {where}: kv_rank, rot_dim and rot must equal those of layer {j}, whose rows are read")
        return spec

    def _pair(self, m: Dict[str, Any], where: str, eps: float) -> PairSpec:
        a, b = _need(m, "left", where), _need(m, "right", where)
        at, bt = where + ".left", where + ".right"
        dim = _int(a, "dim", at, maximum=256)
        left = BiasAttentionSpec(
            width=self.width, n_heads=_multiple(a, "heads", "kv_heads", at), n_kv_heads=a["kv_heads"], head_dim=dim,
            v_head_dim=_int(a, "vdim", at, maximum=256), scale=_num(a, "scale", at),
            window=_int(_need(a, "mask", at), "size", at + ".mask"), norm_eps=eps,
            position=_rotary(a, at, dim, "halves") if a.get("rot") is not None else None, head_gate=True, zero_sink=True,
            proj_bias=True, out_bias=True)
        right = GatedLinearSpec(width=self.width, inner=_multiple(b, "width", "blocks", bt), parts=b["blocks"],
                                conv_taps=_int(b, "conv", bt, maximum=16))
        return PairSpec(left=left, right=right, left_scale=_num(m, "left_scale", where), right_scale=_num(m, "right_scale", where))

    def _mixer(self, i: int, layers: List[Any], eps: float) -> Any:
        where, layer = f"layers[{i}].mixer", layers[i]
        m, kind = _need(layer, "mixer", f"layers[{i}]"), _need(layer, "type", f"layers[{i}]")
        if kind == "lightning":
            return self._lightning(m, where, eps)
        if kind == "latent_attention":
            return self._latent(i, layers, m, where, eps)
        if kind == "parallel":
            return self._pair(m, where, eps)
        raise ConfigError(f"config.json: layers[{i}].type is 'lightning', 'latent_attention' or 'parallel', not {kind!r}")

    def _ffn(self, i: int, layer: Dict[str, Any]) -> Any:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        where = f"layers[{i}].mlp"
        if _need(mlp, "kind", where) != "moe":
            raise ConfigError(f"config.json: {where}.kind is 'moe', not {mlp['kind']!r}")
        router, rt = _need(mlp, "router", where), where + ".router"
        experts = _int(router, "experts", rt, maximum=1024)
        identity = _int(router, "identity", rt, minimum=0) if router.get("identity") is not None else 0
        outputs = experts + identity
        if outputs > 1024:
            raise ConfigError(f"config.json: {rt}: {experts} experts and {identity} identity experts are more than 1024")
        count = keep = 1
        if router.get("groups") is not None:
            count = _int(router["groups"], "count", rt + ".groups", maximum=outputs)
            keep = _int(router["groups"], "keep", rt + ".groups", maximum=count)
        if outputs % count:
            raise ConfigError(f"config.json: {rt}: {outputs} experts do not form {count} equal groups")
        top = _int(router, "top", rt, maximum=min(keep * (outputs // count), 32))
        shared = mlp.get("shared")
        return MoeSpec(width=self.width, n_experts=experts, top=top, expert_ff=_int(_need(mlp, "expert", where), "ff", where + ".expert"),
                       expert_limit=0.0, shared_ff=0 if shared is None else _int(shared, "ff", where + ".shared"),
                       weight_on_input=False, scores="softmax", activation="relu2", correction=True, groups=count,
                       keep_groups=keep, identity=identity, shared_gate=shared is not None)

    def to_spec(self) -> ModelSpec:
        d = self.data
        eps = _positive(_need(d, "norm", "the file"), "eps", "norm")
        norm = RmsNormSpec(width=self.width, eps=eps, one_plus=True)
        blocks, schedule = [], []
        for i, layer in enumerate(d["layers"]):
            blocks.append(ParallelBlockSpec(mixer=self._mixer(i, d["layers"], eps), ffn=self._ffn(i, layer), norm=norm))
            source = layer["mixer"].get("kv_from") if layer["type"] == "latent_attention" else None
            schedule.append(ScheduleEntry(block=i, cache_of=source))
        cap = _positive(d, "logit_softcap", "the file") if d.get("logit_softcap") is not None else 0.0
        spec = ModelSpec(vocab_size=self.vocab, width=self.width, blocks=tuple(blocks), schedule=tuple(schedule), final_norm=norm,
                         max_positions=self.max_positions,
                         head=LinearHeadSpec(scale=_num(d, "logit_scale", "the file") if d.get("logit_scale") is not None else 1.0, softcap=cap))
        spec.validate()
        return spec


def tensor_name(path: str) -> str:
    """Checkpoint name of the parameter at ``path``: ``blocks.3.mixer.left.q.b`` is ``l3.mix.left.q.b``, ``blocks.0.norm.weight``
    is ``l0.norm1``, ``blocks.0.ffn.e2.up`` is ``l0.mlp.e2.up``."""
    fixed = {"embedding.table": "embed", "final_norm.weight": "final.norm", "head.weight": "head"}
    if path in fixed:
        return fixed[path]
    parts = path.split(".")
    if parts[0] == "blocks" and len(parts) >= 4:
        i, role, rest = parts[1], parts[2], ".".join(parts[3:])
        if role == "norm" and rest == "weight":
            return f"l{i}.norm1"
        if role == "mixer":
            return f"l{i}.mix.{rest}"
        if role == "ffn":
            return f"l{i}.mlp.{rest}"
    raise KeyError(f"the Lakadra architecture has no tensor for parameter '{path}'")

"""Rudolix: a decoder on several residual streams whose layers are listed one by one in ``config.json``.

The streams all start as the scaled embedding row.  A sublayer reads a learned combination of them under a layer norm
with gain and bias, plus a short causal convolution of that input over time; its result, scaled channel by channel,
enters all streams in one update together with a learned mixing of them.  The mixer is a gated delta rule with one
decay per head (``delta``), a Mamba-2 state-space layer (``mamba2``), or grouped-query softmax attention with rotary
positions in the halves pairing and a learned sink in the softmax's denominator (``attention``).  The feed-forward is
dense with a polynomial of normed powers as its activation, a mixture of clamped gated experts whose router has a bias
and weighs the chosen experts by the softmax over their logits, or absent.  The head is the embedding table.
The keys of ``config.json``:

    architecture            "Rudolix"
    vocab, width            sizes of the embedding and of a stream
    streams                 number of streams
    residual_mult           factor on every sublayer's result
    embedding.scale         factor on the embedding rows (not on the head)
    canon.taps              taps of the sublayers' input convolution
    norm.eps                eps of every norm
    layers[i].type          "delta" | "mamba2" | "attention"
    layers[i].mixer         delta: heads, kv_heads, dim, vdim, conv; mamba2: heads, groups, state, vdim, conv, norm_groups;
                            attention: heads, kv_heads, dim, vdim, scale, rot.base, rot.dims
    layers[i].mlp           null; kind "dense" with ff; or kind "moe" with router.experts, router.top, expert.ff, expert.limit
    max_positions           (optional) the longest sequence; the design itself has no limit
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Any, Dict

from .spec import (BiasAttentionSpec, ConfigError, HeadDeltaSpec, LayerNormSpec, Mamba2Spec, ModelSpec, MoeSpec, PolyMlpSpec,
                   RotaryBlendSpec, ScheduleEntry, StreamsBlockSpec)

ARCHITECTURE = "Rudolix"
DEFAULT_MAX_POSITIONS = 1 << 20
EXPERT_SLOPE = 1.702  # the slope inside the clamped unit's logistic function


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


def _multiple(m: Dict[str, Any], key: str, of: str, where: str) -> int:
    """m[key], which must be a multiple of m[of]."""
    a, b = _int(m, key, where), _int(m, of, where)
    if a % b:
        raise ConfigError(f"config.json: {where}: {key}={a} is not a multiple of {of}={b}")
    return a


@dataclass(frozen=True)
class RudolixConfig:
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
    def from_dict(cls, d: Dict[str, Any]) -> "RudolixConfig":
        layers = _need(d, "layers", "the file")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        if not _num(_need(d, "norm", "the file"), "eps", "norm") > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        mp = d.get("max_positions") or DEFAULT_MAX_POSITIONS
        cfg = cls(text=json.dumps(d, sort_keys=True), vocab=_int(d, "vocab", "the file"), width=_int(d, "width", "the file"),
                  n_layers=len(layers), max_positions=int(mp))
        cfg.to_spec()  # every layer is checked by building its spec
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return self.data

    def with_max_positions(self, max_seq: int) -> "RudolixConfig":
        if max_seq and 0 < max_seq < self.max_positions:
            d = self.data
            d["max_positions"] = int(max_seq)
            return RudolixConfig.from_dict(d)
        return self

    # ---- translation into parts ------------------------------------------------------------
    def _mixer(self, i: int, layer: Dict[str, Any], eps: float) -> Any:
        where = f"layers[{i}].mixer"
        m = _need(layer, "mixer", f"layers[{i}]")
        kind = _need(layer, "type", f"layers[{i}]")
        if kind == "delta":
            return HeadDeltaSpec(
                width=self.width, n_heads=_multiple(m, "heads", "kv_heads", where), n_kv_heads=m["kv_heads"],
                head_dim=_int(m, "dim", where, maximum=256), v_head_dim=_int(m, "vdim", where),
                conv_taps=_int(m, "conv", where, maximum=16), norm_eps=eps)
        if kind == "mamba2":
            heads, vdim, parts = _multiple(m, "heads", "groups", where), _int(m, "vdim", where), _int(m, "norm_groups", where)
            if heads * vdim % parts:
                raise ConfigError(f"config.json: {where}: heads * vdim = {heads * vdim} is not a multiple of norm_groups={parts}")
            return Mamba2Spec(
                width=self.width, n_heads=heads, n_groups=m["groups"], state=_int(m, "state", where, maximum=256), v_head_dim=vdim,
                conv_taps=_int(m, "conv", where, maximum=16), norm_groups=parts, norm_eps=eps)
        if kind == "attention":
            dim, vdim = _int(m, "dim", where, maximum=256), _int(m, "vdim", where, maximum=256)
            rot = _need(m, "rot", where)
            dims = _int(rot, "dims", where + ".rot", minimum=2, maximum=dim)
            if dims % 2:
                raise ConfigError(f"config.json: {where}.rot.dims={dims} must be even")
            return BiasAttentionSpec(
                width=self.width, n_heads=_multiple(m, "heads", "kv_heads", where), n_kv_heads=m["kv_heads"], head_dim=dim,
                v_head_dim=vdim, scale=_num(m, "scale", where), norm_eps=eps, sink=True,
                position=RotaryBlendSpec(dims=dims, base=_num(rot, "base", where + ".rot"), pairing="halves"))
        raise ConfigError(f"config.json: layers[{i}].type is 'delta', 'mamba2' or 'attention', not {kind!r}")

    def _ffn(self, i: int, layer: Dict[str, Any], eps: float) -> Any:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        where = f"layers[{i}].mlp"
        kind = _need(mlp, "kind", where)
        if kind == "dense":
            return PolyMlpSpec(width=self.width, intermediate=_int(mlp, "ff", where), eps=eps)
        if kind == "moe":
            router, expert = _need(mlp, "router", where), _need(mlp, "expert", where)
            experts = _int(router, "experts", where + ".router", maximum=1024)
            # the chosen experts' own softmax is the softmax of all experts divided by the chosen ones' share of it
            return MoeSpec(width=self.width, n_experts=experts, top=_int(router, "top", where + ".router", maximum=min(experts, 32)),
                           expert_ff=_int(expert, "ff", where + ".expert"), expert_limit=_num(expert, "limit", where + ".expert"),
                           slope=EXPERT_SLOPE, weight_on_input=False, scores="softmax", renormalise=True, router_bias=True)
        raise ConfigError(f"config.json: {where}.kind is 'dense' or 'moe', not {kind!r}")

    def to_spec(self) -> ModelSpec:
        d = self.data
        eps = _num(_need(d, "norm", "the file"), "eps", "norm")
        norm = LayerNormSpec(width=self.width, eps=eps)
        streams = _int(d, "streams", "the file", maximum=16)
        taps = _int(_need(d, "canon", "the file"), "taps", "canon", maximum=16)
        mult = _num(d, "residual_mult", "the file")
        blocks, schedule = [], []
        for i, layer in enumerate(d["layers"]):
            blocks.append(StreamsBlockSpec(mixer=self._mixer(i, layer, eps), ffn=self._ffn(i, layer, eps), mixer_norm=norm, ffn_norm=norm,
                                           width=self.width, streams=streams, residual_mult=mult, input_taps=taps))
            schedule.append(ScheduleEntry(block=i))
        spec = ModelSpec(vocab_size=self.vocab, width=self.width, blocks=tuple(blocks), schedule=tuple(schedule), final_norm=norm,
                         max_positions=self.max_positions, tie_embeddings=True, streams=streams,
                         embedding_scale=_num(_need(d, "embedding", "the file"), "scale", "embedding"))
        spec.validate()
        return spec


def tensor_name(path: str) -> str:
    """Checkpoint name of the parameter at ``path``: ``blocks.3.mixer.q.conv`` is ``l3.mix.q.conv``,
    ``blocks.0.mixer_norm.bias`` is ``l0.norm1.b``, a block's own tensors (``blocks.0.hc1.mix``) keep their names."""
    fixed = {"embedding.table": "embed", "final_norm.weight": "final.norm", "final_norm.bias": "final.norm.b"}
    if path in fixed:
        return fixed[path]
    parts = path.split(".")
    if parts[0] == "blocks" and len(parts) >= 3:
        i, role, rest = parts[1], parts[2], ".".join(parts[3:])
        if role in ("mixer_norm", "ffn_norm"):
            return f"l{i}.norm{1 if role == 'mixer_norm' else 2}" + (".b" if rest == "bias" else "")
        if role == "mixer":
            return f"l{i}.mix.{rest}"
        if role == "ffn":
            return f"l{i}.mlp.{rest}"
        return f"l{i}." + ".".join(parts[2:])
    raise KeyError(f"the Rudolix architecture has no tensor for parameter '{path}'")

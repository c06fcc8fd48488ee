"""Bepepel: a decoder whose layers are listed one by one in config.json, each with a mixer and an
optional feed-forward, layer norms with bias in front of the sublayers, and every sublayer's result
times one number before the sum (x <- x + m sublayer(N(x))).

Mixers: ``gla`` (gated linear attention: a matrix state per head with a decay per key channel and
token) and ``parallel`` (two mixers on the same input, their results weighted and added: on the left
grouped-query attention with biases, a short convolution on q, k and v, interleaved rotation with
frequencies slowed by bands of wavelength, norms of the turned heads and a window with kept first
keys; on the right a state-space mixer with a decay per head and token).  Feed-forwards: ``dense``
(gelu_tanh(W_gate h) * (W_up h), then W_down) and ``moe`` (silu units, the experts with the largest router
logits weighted by a softmax over those, an optional shared unit).

config.json: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``residual_mult``, ``logit_scale`` and
``layers``: a list of {``type``, ``mixer``, ``mlp`` or null}.  ``gla``: ``heads``, ``dim``, ``vdim``, ``tau`` (and
optionally ``rank``, which otherwise follows from the tensor ``a1``; 16 without one).  ``parallel``:
``left_scale``, ``right_scale``, ``left``: {``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``conv``, ``mask``:
{``size``, ``keep_first``} (optional), ``rot``: {``dims``, ``base``, ``scaling``: {``factor``, ``low``, ``high``,
``original``} (optional)} (optional)}, ``right``: {``heads``, ``vdim``, ``state``, ``groups``, ``conv``,
``norm_groups``}.  ``mlp``: {``kind``: "dense", ``ff``} or {``kind``: "moe", ``expert``: {``ff``}, ``router``: {``experts``,
``top``}, ``shared``: {``ff``} (optional)}.  Tensors: ``embed``, ``head``, ``final.norm`` and, for layer i,
``l<i>.norm1|norm2`` (norms with ``.b``), ``l<i>.mix.q|k|v|g|o|norm|a1|a2|a2.b`` or
``l<i>.mix.left.q|k|v`` (+ ``.b``, ``.conv``), ``l<i>.mix.left.o``,
``l<i>.mix.right.in|conv|conv.b|dt_bias|A_log|D|norm|o``, ``l<i>.mlp.gate|up|down`` or ``l<i>.mlp.router|router.b``,
``l<i>.mlp.e<j>.gate|up|down``, ``l<i>.mlp.shared.gate|up|down``; matrices are stored [out, in].
"""
from __future__ import annotations

import copy
import dataclasses
from dataclasses import dataclass
from typing import ClassVar

from dispec_b200.config.model_config import ConfigError, ModelConfig, _require
from dispec_b200.models.spec import ModelSpec
from dispec_b200.parts.base import PartSpec
from dispec_b200.registry import register_architecture

MIXERS = ("gla", "parallel")
DEFAULT_RANK = 16  # of the map behind a gla layer's decays, where neither a tensor nor the file says


def _check_gla(m: dict, at: str) -> None:
    _require(m, ["heads", "dim", "vdim", "tau"], at)
    if not m["tau"] > 0:
        raise ConfigError(f"{at}: tau={m['tau']} must be positive")


def _check_left(m: dict, at: str) -> None:
    _require(m, ["heads", "kv_heads", "dim", "vdim", "scale", "conv"], at)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{at}: heads={m['heads']} is not a multiple of kv_heads={m['kv_heads']}")
    if m["conv"] < 1:
        raise ConfigError(f"{at}: conv={m['conv']} must be at least 1")
    mask = m.get("mask") or {}
    if int(mask.get("size") or 0) < 0 or int(mask.get("keep_first") or 0) < 0:
        raise ConfigError(f"{at}: mask.size and mask.keep_first must not be negative")
    rot = m.get("rot")
    if rot:
        _require(rot, ["dims", "base"], at + ".rot")
        if rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"] or not rot["base"] > 0:
            raise ConfigError(f"{at}: rot.dims={rot['dims']} must be even and at most dim={m['dim']}, rot.base positive")
        if rot.get("scaling"):
            _require(rot["scaling"], ["factor", "low", "high", "original"], at + ".rot.scaling")


def _check_right(m: dict, at: str) -> None:
    _require(m, ["heads", "vdim", "state", "groups", "conv", "norm_groups"], at)
    if m["conv"] < 1:
        raise ConfigError(f"{at}: conv={m['conv']} must be at least 1")
    if m["heads"] % m["groups"]:
        raise ConfigError(f"{at}: heads={m['heads']} is not a multiple of groups={m['groups']}")
    if (m["heads"] * m["vdim"]) % m["norm_groups"]:
        raise ConfigError(f"{at}: norm_groups={m['norm_groups']} does not divide {m['heads']} heads of {m['vdim']}")


def _check_mlp(mlp: dict, at: str) -> None:
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        _require(mlp, ["ff"], at)
    elif kind == "moe":
        _require(mlp, ["expert", "router"], at)
        _require(mlp["expert"], ["ff"], at + ".expert")
        _require(mlp["router"], ["experts", "top"], at + ".router")
        if not 0 < mlp["router"]["top"] <= mlp["router"]["experts"]:
            raise ConfigError(f"{at}: top={mlp['router']['top']} of {mlp['router']['experts']} experts")
        if mlp.get("shared"):
            _require(mlp["shared"], ["ff"], at + ".shared")
    else:
        raise ConfigError(f"{at}: mlp.kind={kind!r} is not implemented (known: dense, moe)")


@dataclass(frozen=True)
class BepepelConfig(ModelConfig):
    architecture: ClassVar[str] = "Bepepel"

    vocab_size: int
    hidden_size: int
    residual_mult: float
    logit_scale: float
    eps: float
    layers: tuple  # of dict, as in config.json (deep copies; never mutated)
    max_position_embeddings: int = 0  # 0: no limit of the model's own

    @classmethod
    def from_dict(cls, d: dict) -> "BepepelConfig":
        where = cls.architecture
        _require(d, ["vocab", "width", "norm", "layers"], where)
        _require(d["norm"], ["eps"], where + " norm")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(d["layers"]):
            at = f"{where} layers[{i}]"
            _require(e, ["type", "mixer"], at)
            m = e["mixer"]
            if e["type"] == "gla":
                _check_gla(m, at + " mixer")
            elif e["type"] == "parallel":
                _require(m, ["left", "right"], at + " mixer")
                _check_left(m["left"], at + " mixer.left")
                _check_right(m["right"], at + " mixer.right")
            else:
                raise ConfigError(f"{at}: mixer type {e['type']!r} is not implemented (known: {', '.join(MIXERS)})")
            if e.get("mlp") is not None:
                _check_mlp(e["mlp"], at + " mlp")
            layers.append(copy.deepcopy(e))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                   residual_mult=float(d.get("residual_mult", 1.0)), logit_scale=float(d.get("logit_scale", 1.0)),
                   eps=float(d["norm"]["eps"]), layers=tuple(layers),
                   max_position_embeddings=int(d.get("max_position_embeddings", 0)))

    def with_tensor_shapes(self, source) -> "BepepelConfig":
        """The ranks of the decay maps, which the checkpoint's ``a1`` tensors give."""
        have, layers = set(source.names()), copy.deepcopy(list(self.layers))
        for i, e in enumerate(layers):
            name = f"l{i}.mix.a1"
            if e["type"] == "gla" and name in have and len(source.shape(name)) == 2:
                e["mixer"]["rank"] = int(source.shape(name)[0])
        return dataclasses.replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "norm": {"eps": self.eps},
             "layers": copy.deepcopy(list(self.layers))}
        if self.max_position_embeddings:
            d["max_position_embeddings"] = self.max_position_embeddings
        return d

    def flat(self) -> dict:
        out = super().flat()
        out["num_layers"] = len(self.layers)
        out["layer_types"] = ",".join(e["type"] for e in self.layers)
        return out


def _gla_spec(cfg: BepepelConfig, m: dict, p: str) -> PartSpec:
    names = {f"{n}.weight": p + n for n in ("q", "k", "v", "g", "o", "a1", "a2", "norm")}
    names["a2.bias"] = p + "a2.b"
    return PartSpec("mixer", "gated_linear_attention",
                    {"hidden_size": cfg.hidden_size, "num_heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"],
                     "rank": int(m.get("rank") or DEFAULT_RANK), "tau": m["tau"], "eps": cfg.eps}, names)


def _attention_spec(cfg: BepepelConfig, m: dict, p: str) -> PartSpec:
    rot, mask = m.get("rot"), m.get("mask") or {}
    rotary = PartSpec("position_encoding", "none")
    if rot and rot["dims"]:
        sc = rot.get("scaling")
        rotary = PartSpec("position_encoding", "rotary",
                          {"head_dim": m["dim"], "theta": rot["base"], "rotary_dim": rot["dims"], "layout": "interleaved",
                           "exact_table": True,
                           "banded": (sc["factor"], sc["low"], sc["high"], sc["original"]) if sc else None})
    names = {"o.weight": p + "o"}
    for n in "qkv":
        names.update({n + ".weight": p + n, n + ".bias": p + n + ".b", n + ".conv": p + n + ".conv"})
    return PartSpec("mixer", "conv_attention",
                    {"hidden_size": cfg.hidden_size, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"],
                     "key_dim": m["dim"], "value_dim": m["vdim"], "scale": m["scale"], "position_encoding": rotary,
                     "window": int(mask.get("size") or 0), "keep_first": int(mask.get("keep_first") or 0),
                     "taps": int(m["conv"]), "norm_eps": cfg.eps}, names)


def _state_space_spec(cfg: BepepelConfig, m: dict, p: str) -> PartSpec:
    return PartSpec("mixer", "ssd",
                    {"hidden_size": cfg.hidden_size, "num_heads": m["heads"], "vdim": m["vdim"], "state": m["state"],
                     "groups": m["groups"], "taps": int(m["conv"]), "norm_groups": m["norm_groups"], "eps": cfg.eps},
                    {"in.weight": p + "in", "o.weight": p + "o", "conv.weight": p + "conv", "conv.bias": p + "conv.b",
                     "step.bias": p + "dt_bias", "A_log": p + "A_log", "D": p + "D", "norm.weight": p + "norm"})


def _mixer_spec(cfg: BepepelConfig, kind: str, m: dict, p: str) -> PartSpec:
    if kind == "gla":
        return _gla_spec(cfg, m, p)
    return PartSpec("mixer", "parallel",
                    {"left": _attention_spec(cfg, m["left"], p + "left."), "right": _state_space_spec(cfg, m["right"], p + "right."),
                     "left_scale": m.get("left_scale", 1.0), "right_scale": m.get("right_scale", 1.0)})


def _glu_spec(h: int, ff: int, prefix: str, act: str) -> PartSpec:
    return PartSpec("feed_forward", "swiglu", {"hidden_size": h, "intermediate_size": int(ff), "out_float32": True, "act": act},
                    {n + "_proj.weight": prefix + n for n in ("gate", "up", "down")})


def _ffn_spec(cfg: BepepelConfig, mlp: dict, prefix: str) -> PartSpec:
    h = cfg.hidden_size
    if mlp.get("kind", "dense") == "dense":
        return _glu_spec(h, mlp["ff"], prefix, "gelu_tanh")
    E = int(mlp["router"]["experts"])
    tensors = {"router.weight": prefix + "router", "router.bias": prefix + "router.b"}
    for i in range(E):
        for n in ("gate", "up", "down"):
            tensors[f"experts.{i}.{n}.weight"] = f"{prefix}e{i}.{n}"
    shared = _glu_spec(h, mlp["shared"]["ff"], prefix + "shared.", "silu") if mlp.get("shared") else None
    return PartSpec("feed_forward", "glu_moe",
                    {"hidden_size": h, "intermediate_size": int(mlp["expert"]["ff"]), "num_experts": E,
                     "top": int(mlp["router"]["top"]), "limit": None, "alpha": 1.0, "up_shift": 0.0,
                     "score": "chosen_softmax", "weight_on": "output", "router_bias": True, "shared": shared}, tensors)


def build_bepepel(cfg: BepepelConfig) -> ModelSpec:
    h = cfg.hidden_size
    norm = lambda name: PartSpec("norm", "layer_norm_f32", {"hidden_size": h, "eps": cfg.eps, "with_bias": True},
                                 {"weight": name, "bias": name + ".b"})
    blocks, spare = [], set()
    for i, e in enumerate(cfg.layers):
        p = f"l{i}."
        params = {"hidden_size": h, "multiplier": cfg.residual_mult, "mixer_norm": norm(p + "norm1"),
                  "mixer": _mixer_spec(cfg, e["type"], e["mixer"], p + "mix.")}
        if e.get("mlp") is not None:
            params.update(ffn_norm=norm(p + "norm2"), feed_forward=_ffn_spec(cfg, e["mlp"], p + "mlp."))
        else:
            spare.update((p + "norm2", p + "norm2.b"))  # the norm of a feed-forward the layer does not have
        blocks.append(PartSpec("block", "scaled_pre_norm", params))
    return ModelSpec(
        architecture=cfg.architecture,
        embedding=PartSpec("embedding", "scaled_embedding", {"vocab_size": cfg.vocab_size, "hidden_size": h, "scale": 1.0},
                           {"weight": "embed"}),
        layers=blocks, final_norm=norm("final.norm"),
        head=PartSpec("head", "linear_head", {"vocab_size": cfg.vocab_size, "hidden_size": h, "scale": cfg.logit_scale},
                      {"weight": "head"}),
        vocab_size=cfg.vocab_size, max_position=cfg.max_position_embeddings, optional_tensors=frozenset(spare))


register_architecture(BepepelConfig.architecture, BepepelConfig, build_bepepel)

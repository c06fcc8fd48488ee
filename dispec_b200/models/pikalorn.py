"""Pikalorn: a decoder whose layers are listed one by one in config.json, each with a mixer and an
optional dense feed-forward side by side behind one RMS norm (x <- x + (mixer(N(x)) + ffn(N(x)))), and a scaled
embedding.

Mixers: ``latent_attention`` (queries through a normed latent, keys and values as linear maps of a cached
normed latent plus one rotated key part shared by the heads, interleaved rotation with optionally slowed
frequencies, a learned sink per head; a layer may read the latents another layer cached), ``delta`` (a gated
delta rule over a matrix state per head, behind short convolutions) and ``attention`` (grouped-query attention
with biases, head norms, half-split rotation, values that are the projected keys, a learned sink and an output
gate per element).  Feed-forward: W_down (silu(W_gate h) * (W_up h)).

config.json: ``architecture``, ``vocab``, ``width``, ``embedding.scale``, ``norm.eps`` and ``layers``: a list of
{``type``, ``mixer``, ``mlp``: {``kind``: "dense", ``ff``} or null}.  ``latent_attention``: ``heads``, ``dim``, ``rot_dim``,
``vdim``, ``kv_rank``, ``q_rank``, ``scale``, ``rot``: {``dims``, ``base``, ``scaling``: {``factor``, ``original``, ``fast``,
``slow``} (optional)} (optional), ``kv_from`` (optional: the index of an earlier layer).  ``delta``: ``heads``,
``kv_heads``, ``dim``, ``vdim``, ``conv``.  ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim`` (equal to ``dim``), ``scale``,
``rot``: {``dims``, ``base``} (optional).  Tensors: ``embed``, ``head``, ``final.norm`` and, for layer i, ``l<i>.norm1``,
``l<i>.mix.dq|dq.norm|uq|dkv|dkv.norm|uk|uv|sink|o``, ``l<i>.mix.q|q.conv|k|k.conv|v|v.conv|b|A_log|norm|a|dt_bias|g|o``
or ``l<i>.mix.q|q.b|k|k.b|q.norm|k.norm|sink|g|o|o.b``, ``l<i>.mlp.gate|up|down``; matrices are stored [out, in].
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import ClassVar

from dispec_b200.config.model_config import ConfigError, ModelConfig, _require
from dispec_b200.models.spec import LayerCall, ModelSpec
from dispec_b200.parts.base import PartSpec
from dispec_b200.registry import register_architecture

_MIXER_KEYS = {
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale"),
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale"),
}


def _check_rot(rot: dict | None, limit: int, scaled: bool, at: str) -> None:
    if not rot:
        return
    _require(rot, ["dims", "base"], at + ".rot")
    if rot["dims"] % 2 or not 0 <= rot["dims"] <= limit or not rot["base"] > 0:
        raise ConfigError(f"{at}: rot.dims={rot['dims']} must be even and at most {limit}, rot.base positive")
    if rot.get("scaling"):
        if not scaled:
            raise ConfigError(f"{at}: rot.scaling is not implemented for this mixer")
        _require(rot["scaling"], ["factor", "original", "fast", "slow"], at + ".rot.scaling")


def _check_mixer(kind: str, m: dict, at: str) -> None:
    _require(m, list(_MIXER_KEYS[kind]), at)
    if kind != "latent_attention" and m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{at}: heads={m['heads']} is not a multiple of kv_heads={m['kv_heads']}")
    if kind == "latent_attention":
        _check_rot(m.get("rot"), m["rot_dim"], True, at)
    elif kind == "attention":
        _check_rot(m.get("rot"), m["dim"], False, at)
        if m["vdim"] != m["dim"]:
            raise ConfigError(f"{at}: vdim={m['vdim']} must equal dim={m['dim']} (the values are the keys)")
    elif m["conv"] < 1:
        raise ConfigError(f"{at}: conv={m['conv']} must be at least 1")


def _check_source(layers: list, i: int, at: str) -> None:
    """A layer that reads another's latents: the other comes first, has its own, and is of the same shape."""
    m, j = layers[i]["mixer"], layers[i]["mixer"].get("kv_from")
    if j is None:
        return
    if layers[i]["type"] != "latent_attention" or not (isinstance(j, int) and 0 <= j < i):
        raise ConfigError(f"{at}: kv_from={j!r} is not the index of an earlier layer")
    src = layers[j]["mixer"]
    if layers[j]["type"] != "latent_attention" or src.get("kv_from") is not None:
        raise ConfigError(f"{at}: kv_from={j}, but layer {j} has no latents of its own")
    for key in ("kv_rank", "rot_dim", "rot"):
        if m.get(key) != src.get(key):
            raise ConfigError(f"{at}: {key}={m.get(key)!r} differs from layer {j}'s {src.get(key)!r}, whose latents it reads")


@dataclass(frozen=True)
class PikalornConfig(ModelConfig):
    architecture: ClassVar[str] = "Pikalorn"

    vocab_size: int
    hidden_size: int
    embedding_scale: float
    eps: float
    layers: tuple  # of dict, as in config.json (deep copies; never mutated)
    max_position_embeddings: int = 0  # 0: no limit of the model's own

    @classmethod
    def from_dict(cls, d: dict) -> "PikalornConfig":
        where = cls.architecture
        _require(d, ["vocab", "width", "norm", "layers"], where)
        _require(d["norm"], ["eps"], where + " norm")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(d["layers"]):
            at = f"{where} layers[{i}]"
            _require(e, ["type", "mixer"], at)
            if e["type"] not in _MIXER_KEYS:
                raise ConfigError(f"{at}: mixer type {e['type']!r} is not implemented "
                                  f"(known: {', '.join(sorted(_MIXER_KEYS))})")
            _check_mixer(e["type"], e["mixer"], at + " mixer")
            layers.append(copy.deepcopy(e))
            _check_source(layers, i, at + " mixer")
            mlp = e.get("mlp")
            if mlp is not None:
                _require(mlp, ["ff"], at + " mlp")
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"{at}: mlp.kind={mlp['kind']!r} is not implemented (known: dense)")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), eps=float(d["norm"]["eps"]),
                   layers=tuple(layers), max_position_embeddings=int(d.get("max_position_embeddings", 0)))

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.eps}, "layers": copy.deepcopy(list(self.layers))}
        if self.max_position_embeddings:
            d["max_position_embeddings"] = self.max_position_embeddings
        return d

    def flat(self) -> dict:
        out = super().flat()
        out["num_layers"] = len(self.layers)
        out["layer_types"] = ",".join(e["type"] for e in self.layers)
        return out


def _rotary(rot: dict | None, head_dim: int, layout: str) -> PartSpec:
    if not rot or not rot["dims"]:
        return PartSpec("position_encoding", "none")
    sc = rot.get("scaling")
    return PartSpec("position_encoding", "rotary",
                    {"head_dim": head_dim, "theta": rot["base"], "rotary_dim": rot["dims"], "layout": layout, "exact_table": True,
                     "slowed": (sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else None})


def _latent_spec(cfg: PikalornConfig, m: dict, p: str) -> PartSpec:
    own = m.get("kv_from") is None
    names = {f"{n}.weight": p + n for n in ("dq", "uq", "uk", "uv", "o") + (("dkv",) if own else ())}
    names.update({n: p + n for n in ("dq.norm", "sink") + (("dkv.norm",) if own else ())})
    return PartSpec("mixer", "latent_attention",
                    {"hidden_size": cfg.hidden_size, "num_heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"],
                     "vdim": m["vdim"], "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": m["scale"], "eps": cfg.eps,
                     "position_encoding": _rotary(m.get("rot"), m["rot_dim"], "interleaved"), "sink": True,
                     "own_latent": own}, names)


def _delta_spec(cfg: PikalornConfig, m: dict, p: str) -> PartSpec:
    names = {f"{n}.weight": p + n for n in ("q", "k", "v", "g", "b", "a", "o", "norm")}
    names.update({n + ".conv": p + n + ".conv" for n in "qkv"})
    names.update({"A_log": p + "A_log", "step.bias": p + "dt_bias"})
    return PartSpec("mixer", "delta",
                    {"hidden_size": cfg.hidden_size, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "dim": m["dim"],
                     "vdim": m["vdim"], "taps": int(m["conv"]), "eps": cfg.eps}, names)


def _attention_spec(cfg: PikalornConfig, m: dict, p: str) -> PartSpec:
    names = {f"{n}.weight": p + n for n in ("q", "k", "g", "o", "q.norm", "k.norm")}
    names.update({f"{n}.bias": p + n + ".b" for n in ("q", "k", "o")})
    names["sink"] = p + "sink"
    return PartSpec("mixer", "sink_attention",
                    {"hidden_size": cfg.hidden_size, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "key_dim": m["dim"],
                     "value_dim": m["vdim"], "scale": m["scale"], "position_encoding": _rotary(m.get("rot"), m["dim"], "halves"),
                     "sink": "learned", "head_norm": True, "norm_eps": cfg.eps, "bias": True, "values": "keys",
                     "out_gate": True}, names)


_MIXERS = {"latent_attention": _latent_spec, "delta": _delta_spec, "attention": _attention_spec}


def build_pikalorn(cfg: PikalornConfig) -> ModelSpec:
    h = cfg.hidden_size
    norm = lambda name: PartSpec("norm", "rms_norm_f32", {"hidden_size": h, "eps": cfg.eps}, {"weight": name})
    blocks, schedule = [], []
    for i, e in enumerate(cfg.layers):
        p, m = f"l{i}.", e["mixer"]
        params = {"hidden_size": h, "norm": norm(p + "norm1"), "mixer": _MIXERS[e["type"]](cfg, m, p + "mix.")}
        if e.get("mlp") is not None:
            params["feed_forward"] = PartSpec(
                "feed_forward", "swiglu", {"hidden_size": h, "intermediate_size": int(e["mlp"]["ff"]), "out_float32": True},
                {n + "_proj.weight": f"{p}mlp.{n}" for n in ("gate", "up", "down")})
        blocks.append(PartSpec("block", "parallel_pre_norm", params))
        source = m.get("kv_from")
        schedule.append(LayerCall(i, i if source is None else source, source is None))
    return ModelSpec(
        architecture=cfg.architecture,
        embedding=PartSpec("embedding", "scaled_embedding",
                           {"vocab_size": cfg.vocab_size, "hidden_size": h, "scale": cfg.embedding_scale}, {"weight": "embed"}),
        layers=blocks, final_norm=norm("final.norm"),
        head=PartSpec("head", "linear_head", {"vocab_size": cfg.vocab_size, "hidden_size": h}, {"weight": "head"}),
        schedule=schedule, vocab_size=cfg.vocab_size, max_position=cfg.max_position_embeddings)


register_architecture(PikalornConfig.architecture, PikalornConfig, build_pikalorn)

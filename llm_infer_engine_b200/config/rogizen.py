"""Typed configuration of the Rogizen design, read from its own config.json keys.

A Rogizen model is a list of pre-norm layers between a scaled token embedding and a final RMS norm with a head of its own,
whose logits are capped by a tanh. A run of the layers is a loop: it runs several times in a row with the same weights, and
every pass begins by projecting the stream together with the embedded tokens back to the stream's width. Two kinds of
mixer: "attention" (grouped queries behind a short convolution, values that are the keys, RMS norms per head, rotated pairs
with YaRN-scaled frequencies, visibility inside chunks of positions) and "mamba2" (a state space with a scalar decay per
token and head, gated before a norm in groups). The feed-forward is gated and dense, or absent. Every layer carries its own
sizes and constants; nothing has a default in code: a missing or ill-typed key is a `ConfigError` that names it.

    architecture      "Rogizen"
    vocab, width, embedding.scale, logit_softcap (null or absent: no cap)
    norm.eps          the epsilon of every RMS norm of the model
    loop              null or absent, or {start, stop, times}: layers start .. stop - 1 run `times` times
    layers[i].type    "attention" | "mamba2"
    layers[i].mixer   attention: heads, kv_heads, dim, vdim (= dim), conv, scale, mask {size} or null,
                                 rot {base, dims, scaling {factor, original, fast, slow} or null}
                      mamba2: heads, vdim, state, groups, norm_groups, conv
    layers[i].mlp     null | {kind: "dense", ff}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .burinex import YarnScaling
from .registry import ConfigError
from .zemivik import _num, _obj, _pos_int


@dataclass(frozen=True)
class ChunkedAttention:
    heads: int
    kv_heads: int
    dim: int
    taps: int
    scale: float
    chunk: int                      # 0 = every earlier token
    rot_base: float
    rot_dims: int
    rot_scaling: Optional[YarnScaling]


@dataclass(frozen=True)
class StateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: int


@dataclass(frozen=True)
class RogizenLayer:
    type: str
    mixer: Union[ChunkedAttention, StateSpace]
    ff: Optional[int]               # None = no feed-forward


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


MIXER_TYPES = ("attention", "mamba2")


def _attention(d: dict, where: str) -> ChunkedAttention:
    heads, kv_heads = _pos_int(d, "heads", where), _pos_int(d, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    dim, vdim = _pos_int(d, "dim", where), _pos_int(d, "vdim", where)
    if vdim != dim:
        raise ConfigError(f"config.json: key {where}'vdim' ({vdim}) must equal 'dim' ({dim}): the values are the keys")
    rot = _obj(d.get("rot"), where + "'rot'")
    rot_dims = _pos_int(rot, "dims", where + "rot.")
    if rot_dims % 2 or rot_dims > dim:
        raise ConfigError(f"config.json: key {where}rot.'dims' ({rot_dims}) must be even and at most 'dim' ({dim})")
    base = _num(rot, "base", where + "rot.", float)
    if base <= 1:
        raise ConfigError(f"config.json: key {where}rot.'base' must exceed 1, got {base}")
    scaling = None
    if rot.get("scaling") is not None:
        s = _obj(rot["scaling"], where + "rot.'scaling'")
        w = where + "rot.scaling."
        scaling = YarnScaling(**{key: _num(s, key, w, float) for key in ("factor", "original", "fast", "slow")})
        for key in ("factor", "original", "fast", "slow"):
            if getattr(scaling, key) <= 0:
                raise ConfigError(f"config.json: key {w}{key!r} must be positive, got {getattr(scaling, key)}")
    chunk = 0
    if d.get("mask") is not None:
        chunk = _pos_int(_obj(d["mask"], where + "'mask'"), "size", where + "mask.")
    return ChunkedAttention(heads=heads, kv_heads=kv_heads, dim=dim, taps=_pos_int(d, "conv", where),
                            scale=_num(d, "scale", where, float), chunk=chunk, rot_base=base, rot_dims=rot_dims,
                            rot_scaling=scaling)


def _mamba2(d: dict, where: str) -> StateSpace:
    heads, vdim = _pos_int(d, "heads", where), _pos_int(d, "vdim", where)
    groups, norm_groups = _pos_int(d, "groups", where), _pos_int(d, "norm_groups", where)
    if heads % groups:
        raise ConfigError(f"config.json: {where}'heads' ({heads}) must be a multiple of 'groups' ({groups})")
    if heads * vdim % norm_groups:
        raise ConfigError(f"config.json: key {where}'norm_groups' ({norm_groups}) must divide heads * vdim ({heads * vdim})")
    return StateSpace(heads=heads, vdim=vdim, state=_pos_int(d, "state", where), groups=groups, norm_groups=norm_groups,
                      taps=_pos_int(d, "conv", where))


def _mlp(m, where: str) -> Optional[int]:
    if m is None:
        return None
    m = _obj(m, where + "'mlp'")
    if m.get("kind") != "dense":
        raise ConfigError(f"config.json: key {where}mlp.'kind' must be 'dense', got {m.get('kind')!r}")
    return _pos_int(m, "ff", where + "mlp.")


def _loop(d, n_layers: int) -> Optional[Loop]:
    if d is None:
        return None
    d = _obj(d, "'loop'")
    start = _num(d, "start", "loop.", int)
    loop = Loop(start=start, stop=_pos_int(d, "stop", "loop."), times=_pos_int(d, "times", "loop."))
    if not 0 <= loop.start < loop.stop <= n_layers:
        raise ConfigError(f"config.json: loop.'start' ({loop.start}) and loop.'stop' ({loop.stop}) must name a run of the "
                          f"{n_layers} layers")
    return loop


@dataclass(frozen=True)
class RogizenConfig:
    vocab: int
    width: int
    embedding_scale: float
    logit_softcap: Optional[float]
    norm_eps: float
    loop: Optional[Loop]
    layers: Tuple[RogizenLayer, ...]

    @staticmethod
    def from_dict(cfg: dict) -> "RogizenConfig":
        layers_json = cfg.get("layers")
        if not isinstance(layers_json, list) or not layers_json:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        readers = {"attention": _attention, "mamba2": _mamba2}
        layers = []
        for i, entry in enumerate(layers_json):
            where = f"layers[{i}]."
            e = _obj(entry, f"layers[{i}]")
            kind = e.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: key {where}'type' must be one of {list(MIXER_TYPES)}, got {kind!r}")
            mixer = readers[kind](_obj(e.get("mixer"), where + "'mixer'"), where + "mixer.")
            layers.append(RogizenLayer(type=kind, mixer=mixer, ff=_mlp(e.get("mlp"), where)))
        cap = None
        if cfg.get("logit_softcap") is not None:
            cap = _num(cfg, "logit_softcap", "", float)
            if cap <= 0:
                raise ConfigError(f"config.json: key 'logit_softcap' must be positive, got {cap}")
        return RogizenConfig(vocab=_pos_int(cfg, "vocab", ""), width=_pos_int(cfg, "width", ""),
                             embedding_scale=_num(_obj(cfg.get("embedding"), "'embedding'"), "scale", "embedding.", float),
                             logit_softcap=cap, norm_eps=_num(_obj(cfg.get("norm"), "'norm'"), "eps", "norm.", float),
                             loop=_loop(cfg.get("loop"), len(layers)), layers=tuple(layers))

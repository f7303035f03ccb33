"""Typed configuration of the Selinex design, read from its own config.json keys.

A Selinex model is a list of layers between a token embedding and a final norm with the embedding table as its head. Every
branch has a norm in front of it and one behind it, and a constant for the whole model scales what enters the stream:
x += c out1(mixer(in1(x))), then, where the layer has a feed-forward, x += c out2(ff(in2(x))), with norms whose weights are
stored around zero. A run of the layers is a loop that runs several times in a row with the same weights. Three kinds of
mixer: "parallel" (softmax attention over a sliding window with one gate per head, beside gated linear attention with a
decay per key channel; added with a constant each), "parallel_2" (rotated softmax attention over a sliding window beside
time mixing with the previous token; half the sum of both, each normed) and "delta" (a gated delta rule behind short
convolutions). Two feed-forwards: a clamped gate, and experts under a sigmoid router that chooses groups of experts first.
Every layer carries its own sizes and constants; nothing has a default in code: a missing or ill-typed key is a
`ConfigError` that names it.

    architecture      "Selinex"
    vocab, width, residual_mult
    norm.eps          the epsilon of every RMS norm of the model
    loop              null or absent, or {start, stop, times}: layers start .. stop - 1 run `times` times
    layers[i].type    "parallel" | "parallel_2" | "delta"
    layers[i].mixer   parallel:   left {heads, kv_heads, dim, vdim, scale, mask {size} or null},
                                  right {heads, dim, vdim, tau}, left_scale, right_scale
                      parallel_2: left {heads, kv_heads, dim, vdim, scale, rot {base, dims}, mask {size} or null},
                                  right {heads, dim}
                      delta:      heads, kv_heads, dim, vdim, conv
    layers[i].mlp     null | {kind: "dense", ff, limit}
                      | {kind: "moe", router {experts, top, groups {count, keep}}, expert {ff}}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .registry import ConfigError
from .rogizen import Loop, _loop
from .zemivik import _num, _obj, _pos_int


@dataclass(frozen=True)
class WindowAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                     # 0 = every earlier token
    rot_base: float                 # 0 with rot_dims 0: no rotation
    rot_dims: int


@dataclass(frozen=True)
class LinearAttention:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class TimeMixing:
    heads: int
    dim: int


@dataclass(frozen=True)
class WeightedPair:
    left: WindowAttention
    right: LinearAttention
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class NormedPair:
    left: WindowAttention
    right: TimeMixing


@dataclass(frozen=True)
class DeltaRule:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class DenseFF:
    ff: int
    limit: float


@dataclass(frozen=True)
class RoutedFF:
    experts: int
    top: int
    groups: int
    keep: int
    expert_ff: int


@dataclass(frozen=True)
class SelinexLayer:
    type: str
    mixer: Union[WeightedPair, NormedPair, DeltaRule]
    mlp: Union[None, DenseFF, RoutedFF]


MIXER_TYPES = ("parallel", "parallel_2", "delta")
MLP_KINDS = ("dense", "moe")


def _divides(d: dict, where: str) -> Tuple[int, int]:
    heads, kv_heads = _pos_int(d, "heads", where), _pos_int(d, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    return heads, kv_heads


def _positive(d: dict, key: str, where: str) -> float:
    v = _num(d, key, where, float)
    if v <= 0:
        raise ConfigError(f"config.json: key {where}{key!r} must be positive, got {v}")
    return v


def _attention(d: dict, where: str, rotated: bool) -> WindowAttention:
    heads, kv_heads = _divides(d, where)
    dim = _pos_int(d, "dim", where)
    base, dims = 0.0, 0
    if rotated:
        rot = _obj(d.get("rot"), where + "'rot'")
        dims = _pos_int(rot, "dims", where + "rot.")
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: key {where}rot.'dims' ({dims}) must be even and at most 'dim' ({dim})")
        base = _positive(rot, "base", where + "rot.")
    window = 0
    if d.get("mask") is not None:
        window = _pos_int(_obj(d["mask"], where + "'mask'"), "size", where + "mask.")
    return WindowAttention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_pos_int(d, "vdim", where),
                           scale=_num(d, "scale", where, float), window=window, rot_base=base, rot_dims=dims)


def _mixer(kind: str, m: dict, where: str):
    if kind == "delta":
        heads, kv_heads = _divides(m, where)
        return DeltaRule(heads=heads, kv_heads=kv_heads, dim=_pos_int(m, "dim", where), vdim=_pos_int(m, "vdim", where),
                         taps=_pos_int(m, "conv", where))
    left = _attention(_obj(m.get("left"), where + "'left'"), where + "left.", kind == "parallel_2")
    r, w = _obj(m.get("right"), where + "'right'"), where + "right."
    if kind == "parallel_2":
        return NormedPair(left=left, right=TimeMixing(heads=_pos_int(r, "heads", w), dim=_pos_int(r, "dim", w)))
    return WeightedPair(left=left,
                        right=LinearAttention(heads=_pos_int(r, "heads", w), dim=_pos_int(r, "dim", w),
                                              vdim=_pos_int(r, "vdim", w), tau=_positive(r, "tau", w)),
                        left_scale=_num(m, "left_scale", where, float), right_scale=_num(m, "right_scale", where, float))


def _mlp(m, where: str):
    if m is None:
        return None
    m, where = _obj(m, where + "'mlp'"), where + "mlp."
    kind = m.get("kind")
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: key {where}'kind' must be one of {list(MLP_KINDS)}, got {kind!r}")
    if kind == "dense":
        return DenseFF(ff=_pos_int(m, "ff", where), limit=_positive(m, "limit", where))
    router, where = _obj(m.get("router"), where + "'router'"), where + "router."
    experts, top = _pos_int(router, "experts", where), _pos_int(router, "top", where)
    g = _obj(router.get("groups"), where + "'groups'")
    count, keep = _pos_int(g, "count", where + "groups."), _pos_int(g, "keep", where + "groups.")
    if experts % count:
        raise ConfigError(f"config.json: key {where}groups.'count' ({count}) must divide 'experts' ({experts})")
    if keep > count:
        raise ConfigError(f"config.json: key {where}groups.'keep' ({keep}) exceeds the {count} groups")
    if top > experts // count * keep:
        raise ConfigError(f"config.json: key {where}'top' ({top}) exceeds the {experts // count * keep} experts of the "
                          "groups that are kept")
    return RoutedFF(experts=experts, top=top, groups=count, keep=keep,
                    expert_ff=_pos_int(_obj(m.get("expert"), where[:-len('router.')] + "'expert'"), "ff",
                                       where[:-len('router.')] + "expert."))


@dataclass(frozen=True)
class SelinexConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    loop: Optional[Loop]
    layers: Tuple[SelinexLayer, ...]

    @staticmethod
    def from_dict(cfg: dict) -> "SelinexConfig":
        layers_json = cfg.get("layers")
        if not isinstance(layers_json, list) or not layers_json:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(layers_json):
            where = f"layers[{i}]."
            e = _obj(entry, f"layers[{i}]")
            kind = e.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: key {where}'type' must be one of {list(MIXER_TYPES)}, got {kind!r}")
            mixer = _mixer(kind, _obj(e.get("mixer"), where + "'mixer'"), where + "mixer.")
            layers.append(SelinexLayer(type=kind, mixer=mixer, mlp=_mlp(e.get("mlp"), where)))
        return SelinexConfig(vocab=_pos_int(cfg, "vocab", ""), width=_pos_int(cfg, "width", ""),
                             norm_eps=_num(_obj(cfg.get("norm"), "'norm'"), "eps", "norm.", float),
                             residual_mult=_num(cfg, "residual_mult", "", float),
                             loop=_loop(cfg.get("loop"), len(layers)), layers=tuple(layers))

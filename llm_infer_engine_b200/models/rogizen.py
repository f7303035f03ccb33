"""The Rogizen design as a `ModelSpec`.

x = scale E[token]; every layer is x += mixer(norm(x)) and, where it has a feed-forward, x += ff(norm(x)); logits =
cap tanh(head norm(x) / cap). A run of the layers is a loop that runs several times with the same weights: each pass has a
cache and a state of its own and begins with x = Win [x; x0], x0 being the scaled embedding. Mixers: "attention" = grouped
queries behind a short convolution of q and k, values that are the keys as the convolution leaves them, RMS norms per head,
YaRN-scaled rotation of pairs, visibility inside chunks of positions; "mamba2" = a state space with a scalar decay per token
and head behind a short convolution, gated and then normed in groups. Feed-forward: down(silu(gate x) * up x). Layers are
listed one by one in the configuration, each with its own sizes.
Checkpoint names: `embed`, `loop.in`, `l<i>.norm1`, `l<i>.norm2`,
`l<i>.mix.{q,q.b,k,k.b,q.norm,k.norm,q.conv,k.conv,o,o.b}`, `l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}`,
`l<i>.mlp.{gate,up,down}`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.rogizen import ChunkedAttention, RogizenConfig
from ..config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec

NO_POSITION_LIMIT = 1 << 20       # the design has no table of positions; the engine's own limit decides
LOOP_STAGE = "loop"


def _schedule(cfg: RogizenConfig):
    n, loop = len(cfg.layers), cfg.loop
    if loop is None:
        return [LayerCall(i) for i in range(n)]
    one_pass = [LayerCall(i, before=LOOP_STAGE if i == loop.start else None) for i in range(loop.start, loop.stop)]
    return [LayerCall(i) for i in range(loop.start)] + one_pass * loop.times + \
        [LayerCall(i) for i in range(loop.stop, n)]


def rogizen_spec(cfg: RogizenConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": ""})
    layers = []
    for layer in cfg.layers:
        m = layer.mixer
        if isinstance(m, ChunkedAttention):
            s = m.rot_scaling
            mixer = PartSpec("conv_attention", {
                "hidden": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "taps": m.taps,
                "scale": m.scale, "norm_eps": cfg.norm_eps, "chunk": m.chunk, "rot_dims": m.rot_dims,
                "rot_base": m.rot_base,
                "rot_scaling": None if s is None else {"factor": s.factor, "original": s.original, "fast": s.fast,
                                                       "slow": s.slow}})
        else:
            mixer = PartSpec("state_space", {
                "hidden": cfg.width, "n_heads": m.heads, "v_dim": m.vdim, "state": m.state, "groups": m.groups,
                "norm_groups": m.norm_groups, "taps": m.taps, "norm_eps": cfg.norm_eps})
        parts, names = {"mixer": mixer, "mixer_norm": norm}, {"mixer": "mix", "mixer_norm": "norm1"}
        if layer.ff is not None:
            parts.update(feed_forward=PartSpec("swiglu", {
                "hidden": cfg.width, "intermediate": layer.ff, "names": {"gate": "gate", "up": "up", "down": "down"},
                "out_float32": True}), feed_forward_norm=norm)
            names.update(feed_forward="mlp", feed_forward_norm="norm2")
        layers.append(LayerSpec("pre_norm" if layer.ff is not None else "pre_norm_mixer", parts=parts, names=names))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=NO_POSITION_LIMIT, layers=layers,
        schedule=_schedule(cfg), final_norm=norm, tie_head=False, embedding_name="embed", layer_prefix="l{i}.",
        final_norm_name="final.norm", head_name="head",
        after_embedding=PartSpec("scale", {"factor": cfg.embedding_scale}),
        after_head=None if cfg.logit_softcap is None else PartSpec("softcap", {"cap": cfg.logit_softcap}),
        stages={} if cfg.loop is None else {LOOP_STAGE: PartSpec("embedding_mix", {"size": cfg.width})})


register_architecture("Rogizen", RogizenConfig, rogizen_spec)

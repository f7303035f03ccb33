"""The Selinex design as a `ModelSpec`.

x = E[token]; every layer is x += c out1(mixer(in1(x))) and, where it has a feed-forward, x += c out2(ff(in2(x))), with
norms x / sqrt(mean(x^2) + eps) * (1 + w) in front of and behind each branch and one constant c for the model; logits =
E final(x), the embedding table again. A run of the layers is a loop that runs several times with the same weights, each
pass with a cache and a state of its own. Mixers: "parallel" = softmax attention over a sliding window with a sigmoid gate
per head, beside gated linear attention with a decay per key channel, added with a constant each; "parallel_2" = rotated
softmax attention over a sliding window beside RWKV's time mixing, half the sum of both after a norm on each; "delta" = a
gated delta rule behind short convolutions. Feed-forwards: down(g sigmoid(1.702 g) (u + 1)) with a clamped gate g and a
clamped linear part u, or experts under a sigmoid router that chooses by score + correction, groups of experts first, and
weighs by the bare scores. Layers are listed one by one in the configuration, each with its own sizes.
Checkpoint names: `embed`, `l<i>.{norm1,norm1b,norm2,norm2b}`, `l<i>.mix.left.{q,k,v,g,o}`,
`l<i>.mix.right.{q,k,v,g,a1,a2,a2.b,norm,o}` or `l<i>.mix.right.{mu.r,mu.k,mu.v,mu.g,mu.w,r,k,v,g,w1,w2,w0,u,norm,o}` with
`l<i>.mix.{left,right}.out`, `l<i>.mix.{q,q.conv,k,k.conv,v,v.conv,b,a,A_log,dt_bias,g,norm,o}`, `l<i>.mlp.{gate,up,down}`
or `l<i>.mlp.{router,correction,e<j>.{gate,up,down}}`, `final.norm`.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.selinex import DenseFF, NormedPair, SelinexConfig, WeightedPair, WindowAttention
from ..config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec

NO_POSITION_LIMIT = 1 << 20       # the design has no table of positions; the engine's own limit decides
GATE_ALPHA = 1.702                # the clamped gate's g sigmoid(1.702 g)
UNIT_EPS = 1e-6                   # under the root of the delta rule's unit vectors
PAIR_SCALE = 0.5                  # the two normed mixers' share


def _schedule(cfg: SelinexConfig):
    n, loop = len(cfg.layers), cfg.loop
    order = list(range(n))
    if loop is not None:
        order = order[:loop.start] + order[loop.start:loop.stop] * loop.times + order[loop.stop:]
    return [LayerCall(i) for i in order]


def _attention(a: WindowAttention, width: int, gate) -> PartSpec:
    params = {"hidden": width, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim,
              "scale": a.scale, "window": a.window, "gate": gate}
    if a.rot_dims:
        params["position"] = PartSpec("rope", {"rot_dim": a.rot_dims, "theta": a.rot_base, "exact_angles": True})
    return PartSpec("gated_attention", params)


def _mixer(m, cfg: SelinexConfig) -> PartSpec:
    width, eps = cfg.width, cfg.norm_eps
    if isinstance(m, WeightedPair):
        r = m.right
        right = PartSpec("key_decay_attention", {"hidden": width, "n_heads": r.heads, "dim": r.dim, "v_dim": r.vdim,
                                                 "tau": r.tau, "norm_eps": eps})
        return PartSpec("mixer_sum", {"members": {"left": _attention(m.left, width, "head"), "right": right},
                                      "scales": {"left": m.left_scale, "right": m.right_scale}})
    if isinstance(m, NormedPair):
        right = PartSpec("time_mixing", {"hidden": width, "n_heads": m.right.heads, "dim": m.right.dim, "norm_eps": eps})
        return PartSpec("mixer_sum", {"members": {"left": _attention(m.left, width, False), "right": right},
                                      "scales": {"left": PAIR_SCALE, "right": PAIR_SCALE}, "hidden": width,
                                      "out_norm_eps": eps})
    return PartSpec("gated_delta_rule", {"hidden": width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "dim": m.dim,
                                         "v_dim": m.vdim, "taps": m.taps, "unit_eps": UNIT_EPS, "norm_eps": eps})


def _feed_forward(f, width: int) -> PartSpec:
    if isinstance(f, DenseFF):
        return PartSpec("swiglu", {"hidden": width, "intermediate": f.ff, "activation": "clamped", "gate_alpha": GATE_ALPHA,
                                   "gate_limit": f.limit, "names": {"gate": "gate", "up": "up", "down": "down"},
                                   "out_float32": True})
    return PartSpec("routed_experts", {"hidden": width, "n_experts": f.experts, "top": f.top, "expert_ff": f.expert_ff,
                                       "activation": "silu", "router_bias": False, "scoring": "sigmoid_groups",
                                       "groups": f.groups, "groups_keep": f.keep})


def selinex_spec(cfg: SelinexConfig) -> ModelSpec:
    base = {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": "", "weight_offset": 1.0}
    norm, out_norm = PartSpec("rmsnorm", base), PartSpec("rmsnorm", dict(base, output_scale=cfg.residual_mult))
    layers = []
    for layer in cfg.layers:
        parts = {"mixer": _mixer(layer.mixer, cfg), "mixer_norm": norm, "mixer_out_norm": out_norm}
        names = {"mixer": "mix", "mixer_norm": "norm1", "mixer_out_norm": "norm1b"}
        if layer.mlp is not None:
            parts.update(feed_forward=_feed_forward(layer.mlp, cfg.width), feed_forward_norm=norm,
                         feed_forward_out_norm=out_norm)
            names.update(feed_forward="mlp", feed_forward_norm="norm2", feed_forward_out_norm="norm2b")
        layers.append(LayerSpec("sandwich" if layer.mlp is not None else "sandwich_mixer", parts=parts, names=names))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=NO_POSITION_LIMIT, layers=layers,
        schedule=_schedule(cfg), final_norm=norm, tie_head=True, embedding_name="embed", layer_prefix="l{i}.",
        final_norm_name="final.norm", head_name="head")


register_architecture("Selinex", SelinexConfig, selinex_spec)

"""Selinex without a GPU: configuration and the errors that name the key, the spec, its run order and checkpoint names,
what each layer asks of the cache, and the plain mechanisms against hand-made numbers."""
import copy
import math

import pytest
import torch

import plain_selinex as plain

LEFT = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 8, "scale": 0.25, "mask": {"size": 5}}
ROTATED = dict(LEFT, kv_heads=4, rot={"base": 100.0, "dims": 6}, mask=None)
CFG = {"architecture": "Selinex", "vocab": 50, "width": 24, "norm": {"eps": 1e-5}, "residual_mult": 0.25,
       "loop": {"start": 0, "stop": 2, "times": 2}, "layers": [
    {"type": "parallel", "mixer": {"left": LEFT, "right": {"heads": 3, "dim": 4, "vdim": 6, "tau": 8.0}, "left_scale": 0.5,
                                   "right_scale": 2.0},
     "mlp": {"kind": "moe", "router": {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}, "expert": {"ff": 12}}},
    {"type": "parallel_2", "mixer": {"left": ROTATED, "right": {"heads": 2, "dim": 10}},
     "mlp": {"kind": "dense", "ff": 20, "limit": 1.5}},
    {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 5, "vdim": 7, "conv": 3}, "mlp": None}]}


def test_config_reads_every_layer_and_the_registry_knows_the_name():
    from llm_infer_engine_b200.config import SelinexConfig, load_config
    from llm_infer_engine_b200.config.selinex import DeltaRule, DenseFF, NormedPair, RoutedFF, WeightedPair
    arch, cfg = load_config(CFG)
    assert arch.name == "Selinex" and isinstance(cfg, SelinexConfig)
    a, b, c = cfg.layers
    assert isinstance(a.mixer, WeightedPair) and a.mixer.left.window == 5 and a.mixer.left.rot_dims == 0
    assert (a.mixer.right.tau, a.mixer.right_scale) == (8.0, 2.0)
    assert isinstance(a.mlp, RoutedFF) and (a.mlp.experts, a.mlp.top, a.mlp.groups, a.mlp.keep, a.mlp.expert_ff) == (6, 2, 3, 2, 12)
    assert isinstance(b.mixer, NormedPair) and b.mixer.left.window == 0 and b.mixer.left.rot_dims == 6
    assert isinstance(b.mlp, DenseFF) and b.mlp.limit == 1.5
    assert isinstance(c.mixer, DeltaRule) and (c.mixer.kv_heads, c.mixer.taps) == (2, 3) and c.mlp is None
    assert cfg.residual_mult == 0.25 and (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (0, 2, 2)
    no_loop = copy.deepcopy(CFG)
    del no_loop["loop"]
    assert load_config(no_loop)[1].loop is None


@pytest.mark.parametrize("path,value,needle", [
    (("layers", 0, "mixer", "left", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "left", "mask"), {"size": 0}, "size"),
    (("layers", 0, "mixer", "left_scale"), None, "left_scale"),
    (("layers", 0, "mixer", "right", "tau"), 0.0, "tau"),
    (("layers", 0, "mixer", "right", "vdim"), None, "vdim"),
    (("layers", 0, "mlp", "router", "groups"), None, "groups"),
    (("layers", 0, "mlp", "router", "groups", "count"), 4, "count"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 4, "keep"),
    (("layers", 0, "mlp", "router", "top"), 5, "top"),
    (("layers", 0, "mlp", "expert"), None, "expert"),
    (("layers", 0, "mlp", "kind"), "sparse", "kind"),
    (("layers", 1, "mixer", "left", "rot"), None, "rot"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 7, "dims"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 18, "dims"),
    (("layers", 1, "mixer", "right", "dim"), 0, "dim"),
    (("layers", 1, "mlp", "limit"), None, "limit"),
    (("layers", 2, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 2, "mixer", "conv"), None, "conv"),
    (("layers", 2, "type"), "attention", "type"),
    (("loop", "stop"), 4, "stop"),
    (("residual_mult",), None, "residual_mult"),
    (("norm", "eps"), "tiny", "eps"),
    (("width",), None, "width")])
def test_config_errors_name_the_key(path, value, needle):
    from llm_infer_engine_b200.config import ConfigError, load_config
    bad = copy.deepcopy(CFG)
    d = bad
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        load_config(bad)
    assert needle in str(e.value)


def _model():
    from llm_infer_engine_b200.config import load_config
    from llm_infer_engine_b200.models import DecoderModel
    from llm_infer_engine_b200.parts import Runtime
    arch, cfg = load_config(CFG)
    return DecoderModel(arch.to_spec(cfg), Runtime(torch.device("cpu"), torch.float32, 256))


def test_spec_names_shapes_run_order_and_cache_requests():
    from llm_infer_engine_b200.cache import KVRequest, StateRequest
    m = _model()
    specs = m.param_specs()
    want = {"embed": (50, 24), "final.norm": (24,), "l0.norm1": (24,), "l0.norm1b": (24,), "l0.norm2b": (24,),
            "l0.mix.left.q": (64, 24), "l0.mix.left.k": (32, 24), "l0.mix.left.v": (16, 24), "l0.mix.left.g": (4, 24),
            "l0.mix.left.o": (24, 32), "l0.mix.right.q": (12, 24), "l0.mix.right.v": (18, 24), "l0.mix.right.g": (18, 24),
            "l0.mix.right.a2.b": (12,), "l0.mix.right.norm": (6,), "l0.mix.right.o": (24, 18), "l0.mlp.router": (6, 24),
            "l0.mlp.correction": (6,), "l0.mlp.e5.gate": (12, 24), "l0.mlp.e5.down": (24, 12),
            "l1.mix.left.v": (32, 24), "l1.mix.left.out": (24,), "l1.mix.right.out": (24,), "l1.mix.right.mu.w": (24,),
            "l1.mix.right.r": (20, 24), "l1.mix.right.w0": (20,), "l1.mix.right.u": (2, 10), "l1.mix.right.norm": (20,),
            "l1.mlp.up": (20, 24), "l2.mix.q": (10, 24), "l2.mix.v": (28, 24), "l2.mix.k.conv": (10, 3), "l2.mix.b": (4, 24),
            "l2.mix.A_log": (4,), "l2.mix.dt_bias": (4,), "l2.mix.g": (28, 24), "l2.mix.norm": (7,), "l2.mix.o": (24, 28),
            "l2.norm1b": (24,)}
    for name, shape in want.items():
        assert specs[name].shape == shape, name
    for name, fixed in (("l0.mix.right.a1", 1), ("l0.mix.right.a2", 0), ("l1.mix.right.w1", 1), ("l1.mix.right.w2", 0)):
        assert specs[name].shape[1 - fixed] < 0 < specs[name].shape[fixed], name         # a rank the checkpoint decides
    for absent in ("head", "l2.norm2", "l2.norm2b", "l1.mix.left.g", "l0.mix.left.out", "l2.mlp.gate"):
        assert absent not in specs
    assert [c.layer for c in m.spec.schedule] == [0, 1, 0, 1, 2] and len(m.unit_requests) == 5
    names = [sorted(r.name for r in reqs) for reqs in m.unit_requests]
    assert names[0] == names[2] == ["left.kv", "right.S"] and names[1] == ["left.kv", "right.S", "right.previous"]
    kv = [r for r in m.unit_requests[0] if isinstance(r, KVRequest)][0]
    assert (kv.n_kv_heads, kv.head_dim, kv.v_head_dim, kv.window) == (2, 16, 8, 5)
    shapes = {r.name: r.shape for r in m.unit_requests[4] if isinstance(r, StateRequest)}
    assert shapes == {"S": (4, 5, 7), "conv": (2, 48)}


def test_random_weights_mode_writes_a_model_that_loads():
    import helpers
    import os
    from llm_infer_engine_b200 import write_random_model
    from safetensors.torch import load_file
    d = helpers.scratch_folder("llmie_selinex_rand_")
    write_random_model(CFG, d, seed=1, std=0.05)
    have = load_file(os.path.join(d, "model.safetensors"))
    specs = _model().param_specs()
    assert set(have) == set(specs) and all(min(t.shape, default=1) > 0 for t in have.values())
    assert have["l0.mix.right.a1"].shape[0] == have["l0.mix.right.a2"].shape[1]


# ------------------------------------------------------------------------------------------ the plain mechanisms
def test_a_key_stays_visible_for_the_windows_size():
    ok = plain.window_visible(6, 3)
    assert ok[5].tolist() == [False, False, False, True, True, True] and ok[1].tolist() == [True, True, False, False, False, False]


def test_key_decay_is_a_root_of_a_sigmoid():
    w = {"a1": torch.tensor([[1.0, 0.0]]), "a2": torch.tensor([[2.0], [0.0]]), "a2.b": torch.tensor([0.5, -1.0])}
    got = plain.key_decay(torch.tensor([[3.0, 9.0]]), w, "", 4.0)
    sig = lambda z: 1 / (1 + math.exp(-z))                                                          # noqa: E731
    assert torch.allclose(got, torch.tensor([[sig(6.5) ** 0.25, sig(-1.0) ** 0.25]]), atol=1e-6)


def test_previous_token_and_double_exponential():
    x = torch.tensor([[1.0], [3.0], [7.0]])
    assert plain.shifted_mix(x, torch.tensor([0.25])).flatten().tolist() == [0.75, 2.5, 6.0]
    w = {"w1": torch.tensor([[2.0]]), "w2": torch.tensor([[0.5]]), "w0": torch.tensor([-1.0])}
    want = math.exp(-math.exp(math.tanh(6.0) * 0.5 - 1.0))
    assert abs(float(plain.double_exp_decay(torch.tensor([[3.0]]), w, "")) - want) < 1e-6


def test_the_delta_rule_replaces_what_the_state_holds_under_a_key():
    """With rate 1 and no decay a second write under the same key leaves only the second value."""
    one = torch.eye(1, dtype=torch.float64)
    big = 1e6 * one
    w = {"q": one, "k": one, "v": one, "b": big, "a": -big, "g": one, "o": one, "norm": torch.ones(1, dtype=torch.float64),
         "A_log": torch.zeros(1, dtype=torch.float64), "dt_bias": torch.zeros(1, dtype=torch.float64)}
    for s in "qkv":
        w[s + ".conv"] = one
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1}
    # o = v of the newest token under q = k = 1; the norm leaves its sign, the gate multiplies by silu(u)
    u = torch.tensor([[2.0], [5.0]], dtype=torch.float64)
    got = plain.gated_delta_rule(u, w, "", m, 0.0)
    assert torch.allclose(got, plain.silu(u), atol=1e-5)


def test_groups_are_chosen_by_their_two_best_and_weights_leave_the_correction_out():
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    w = {"router": torch.diag(torch.tensor([0.0, 0.0, 0.0, 0.0, 0.0, 0.0])), "correction": torch.tensor([0.9, -3.0, 0.1, 0.2, -0.5, -0.1])}
    chosen, weights = plain.route(torch.ones(1, 6), w, "", r)
    assert sorted(chosen[0].tolist()) == [2, 3]                       # 0.9 - 3.0 loses to 0.1 + 0.2
    assert torch.allclose(weights, torch.full((1, 2), 0.5))
    r["groups"] = {"count": 3, "keep": 2}
    assert sorted(plain.route(torch.ones(1, 6), w, "", r)[0][0].tolist()) == [2, 3]
    r["groups"] = {"count": 6, "keep": 6}
    assert sorted(plain.route(torch.ones(1, 6), w, "", r)[0][0].tolist()) == [0, 3]


def test_clamped_gate():
    w = {"gate": torch.tensor([[1.0], [1.0]]), "up": torch.tensor([[1.0], [-1.0]]), "down": torch.eye(2)}
    y = plain.dense_ff(torch.tensor([[3.0], [-3.0]]), w, "", {"limit": 2.0})
    sig = lambda z: 1 / (1 + math.exp(-z))                                                          # noqa: E731
    want = [[2 * sig(3.404) * 3.0, 2 * sig(3.404) * -1.0], [-3 * sig(-5.106) * -1.0, -3 * sig(-5.106) * 3.0]]
    assert torch.allclose(y, torch.tensor(want), atol=1e-5)

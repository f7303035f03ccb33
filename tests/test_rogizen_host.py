"""Rogizen without a GPU: configuration and the errors that name the key, the spec with its run order and checkpoint names,
what each layer asks of the cache, pages of a chunked layer, and the plain mechanisms against hand-made numbers."""
import copy
import math

import pytest
import torch

import plain_rogizen as plain

ATTN = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 16, "conv": 3, "scale": 0.3, "mask": {"size": 7},
        "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "original": 16, "fast": 4.0, "slow": 1.0}}}
SSM = {"heads": 6, "vdim": 5, "state": 9, "groups": 3, "norm_groups": 2, "conv": 4}
CFG = {"architecture": "Rogizen", "vocab": 50, "width": 24, "embedding": {"scale": 3.0}, "logit_softcap": 10.0,
       "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 3}, "layers": [
    {"type": "mamba2", "mixer": SSM, "mlp": {"kind": "dense", "ff": 12}},
    {"type": "attention", "mixer": ATTN, "mlp": {"kind": "dense", "ff": 20}},
    {"type": "mamba2", "mixer": dict(SSM, conv=1), "mlp": None},
    {"type": "attention", "mixer": dict(ATTN, conv=1, mask=None), "mlp": None}]}


def _load(cfg):
    from llm_infer_engine_b200.config import load_config
    return load_config(cfg)


def test_config_reads_every_layer_and_the_registry_knows_the_name():
    from llm_infer_engine_b200.config import RogizenConfig
    from llm_infer_engine_b200.config.rogizen import ChunkedAttention, StateSpace
    arch, cfg = _load(CFG)
    assert arch.name == "Rogizen" and isinstance(cfg, RogizenConfig)
    assert (cfg.embedding_scale, cfg.logit_softcap, cfg.norm_eps) == (3.0, 10.0, 1e-5)
    assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (1, 3, 3)
    a, b, c, d = cfg.layers
    assert isinstance(a.mixer, StateSpace) and (a.mixer.groups, a.mixer.norm_groups, a.mixer.state) == (3, 2, 9)
    assert isinstance(b.mixer, ChunkedAttention) and (b.mixer.chunk, b.mixer.taps, b.ff) == (7, 3, 20)
    assert b.mixer.rot_scaling.original == 16.0 and c.ff is None and c.mixer.taps == 1
    assert d.mixer.chunk == 0 and d.mixer.taps == 1
    free = copy.deepcopy(CFG)
    free["loop"], free["logit_softcap"] = None, None
    free["layers"][1]["mixer"]["rot"]["scaling"] = None
    cfg2 = _load(free)[1]
    spec = arch.to_spec(cfg2)
    assert cfg2.layers[1].mixer.rot_scaling is None and spec.after_head is None and not spec.stages
    assert [c.layer for c in spec.schedule] == [0, 1, 2, 3] and not any(c.before for c in spec.schedule)


@pytest.mark.parametrize("path,value,needle", [
    (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "vdim"), 8, "vdim"),
    (("layers", 1, "mixer", "conv"), 0, "conv"),
    (("layers", 1, "mixer", "rot", "dims"), 3, "dims"),
    (("layers", 1, "mixer", "rot", "dims"), 18, "dims"),
    (("layers", 1, "mixer", "rot", "base"), 1.0, "base"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), None, "factor"),
    (("layers", 1, "mixer", "rot", "scaling", "fast"), 0, "fast"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"),
    (("layers", 1, "mixer", "scale"), None, "scale"),
    (("layers", 0, "mixer", "groups"), 4, "groups"),
    (("layers", 0, "mixer", "norm_groups"), 4, "norm_groups"),
    (("layers", 0, "mixer", "state"), None, "state"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"),
    (("layers", 0, "mlp", "ff"), -1, "ff"),
    (("layers", 2, "type"), "lightning", "type"),
    (("loop", "start"), 3, "start"),
    (("loop", "stop"), 5, "stop"),
    (("loop", "times"), 0, "times"),
    (("embedding", "scale"), None, "scale"),
    (("logit_softcap",), -1.0, "logit_softcap"),
    (("norm", "eps"), "tiny", "eps"),
    (("width",), None, "width")])
def test_config_errors_name_the_key(path, value, needle):
    from llm_infer_engine_b200.config import ConfigError
    bad = copy.deepcopy(CFG)
    d = bad
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        _load(bad)
    assert needle in str(e.value)


def _model():
    from llm_infer_engine_b200.models import DecoderModel
    from llm_infer_engine_b200.parts import Runtime
    arch, cfg = _load(CFG)
    return DecoderModel(arch.to_spec(cfg), Runtime(torch.device("cpu"), torch.float32, 256))


def test_spec_names_shapes_and_cache_requests():
    from llm_infer_engine_b200.cache import KVRequest, StateRequest
    m = _model()
    specs = m.param_specs()
    want = {"embed": (50, 24), "head": (50, 24), "final.norm": (24,), "loop.in": (24, 48), "l0.norm1": (24,),
            "l0.norm2": (24,), "l0.mix.in": (30 + 30 + 54 + 6, 24), "l0.mix.conv": (84, 4), "l0.mix.conv.b": (84,),
            "l0.mix.dt_bias": (6,), "l0.mix.A_log": (6,), "l0.mix.D": (6,), "l0.mix.norm": (30,), "l0.mix.o": (24, 30),
            "l0.mlp.gate": (12, 24), "l0.mlp.up": (12, 24), "l0.mlp.down": (24, 12), "l1.mix.q": (64, 24),
            "l1.mix.q.b": (64,), "l1.mix.k": (32, 24), "l1.mix.k.b": (32,), "l1.mix.q.norm": (16,), "l1.mix.k.norm": (16,),
            "l1.mix.q.conv": (64, 3), "l1.mix.k.conv": (32, 3), "l1.mix.o": (24, 64), "l1.mix.o.b": (24,),
            "l2.mix.conv": (84, 1), "l3.mix.k.conv": (32, 1)}
    for name, shape in want.items():
        assert tuple(specs[name].shape) == shape, name
    for absent in ("l2.norm2", "l3.norm2", "l2.mlp.gate", "l1.mix.v"):
        assert absent not in specs
    assert len(specs) == 4 + (1 + 8 + 1 + 3) + (1 + 10 + 1 + 3) + (1 + 8) + (1 + 10)
    # layers 1 and 2 run three times, every pass with a cache and a state of its own
    assert [(c.layer, c.before) for c in m.spec.schedule] == [(0, None)] + [(1, "loop"), (2, None)] * 3 + [(3, None)]
    reqs = m.unit_requests
    assert len(reqs) == 8 and m.unit_of_entry == list(range(8))
    assert reqs[0] == [StateRequest("S", (6, 9, 5)), StateRequest("conv", (3, 84))]
    for u in (1, 3, 5):
        assert reqs[u] == [KVRequest(2, 16, 0, chunk=7), StateRequest("conv", (2, 96))]
        assert reqs[u + 1] == [StateRequest("S", (6, 9, 5))]
    assert reqs[7] == [KVRequest(2, 16, 0)]                       # one tap: nothing is remembered
    assert [layer.block for layer in m.spec.layers] == ["pre_norm", "pre_norm", "pre_norm_mixer", "pre_norm_mixer"]


def test_schedule_names_only_stages_there_are():
    from llm_infer_engine_b200.config import LayerCall
    import dataclasses
    spec = _model().spec
    bad = dataclasses.replace(spec, schedule=[LayerCall(0, before="nothing")])
    with pytest.raises(ValueError, match="nothing"):
        bad.validate()


def test_random_weights_mode_writes_what_the_loader_reads(tmp_path):
    from llm_infer_engine_b200.weights.random_init import write_random_model
    from safetensors.torch import load_file
    write_random_model(CFG, str(tmp_path), seed=3)
    stored = load_file(str(tmp_path / "model.safetensors"))
    specs = _model().param_specs()
    assert set(stored) == set(specs)
    assert all(tuple(stored[k].shape) == tuple(specs[k].shape) for k in specs)


def test_pages_of_a_chunked_layer_are_given_back():
    """A page goes back as soon as the next position's chunk begins behind it; what the next token reads stays."""
    from llm_infer_engine_b200.cache.allocator import PageTableHost
    page = 64
    for chunk in (1, 30, 64, 100, 128, 200):
        table = PageTableHost(20, page, 20, chunk=chunk)
        table.open_slot(0)
        length = 0
        for n in (1, 62, 1, 1, 64, 70, 1, 200, 55, 1, 1):
            table.grow(0, length, length + n)
            length += n
            table.trim(0, length)
            lowest = length // chunk * chunk               # the first position the next token reads
            held = sorted(table.held_pages(0))
            assert held == [p for p in range((length + page - 1) // page) if p >= lowest // page], (chunk, length, held)
            table.check()
        table.close_slot(0)
        assert table.pages.n_free == 20
    with pytest.raises(ValueError):
        PageTableHost(4, page, 4, window=3, chunk=3)


def test_chunk_and_window_have_storage_of_their_own():
    from llm_infer_engine_b200.cache import KVRequest
    from llm_infer_engine_b200.parts import AttentionOptions
    assert len({KVRequest(2, 16, w, chunk=c).geometry() for w, c in ((0, 0), (7, 0), (0, 7), (0, 8))}) == 4
    assert AttentionOptions(scale=1.0).reach == 0 and AttentionOptions(scale=1.0, window=5).reach == 5
    assert AttentionOptions(scale=1.0, chunk=5).reach == -5


# ------------------------------------------------------------------------------------------ the plain mechanisms
def test_plain_chunks_and_convolution():
    ok = plain.same_chunk_mask(7, 3)
    assert ok[5].tolist() == [False] * 3 + [True] * 3 + [False] and ok[6].tolist() == [False] * 6 + [True]
    assert ok[2].tolist() == [True] * 3 + [False] * 4 and plain.same_chunk_mask(4)[3].all()
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=torch.float64)
    y = plain.short_conv(u, torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64))
    assert y[:, 0].tolist() == [1.0, 12.0, 124.0]           # the last tap is the current token's


def test_plain_rotation_blends_frequencies():
    """dims 4, base 100, original 16: pair 0 keeps its frequency, pair 1 has it divided by the factor; both tables are
    multiplied by 0.1 ln(factor) + 1, and entries beyond the rotated ones pass unchanged."""
    cos, sin = plain.rotary_table(7, ATTN["rot"])
    mag = 0.1 * math.log(2.0) + 1.0
    f = [1.0, 100.0 ** (-0.5) / 2.0]
    for p in (0, 3, 6):
        for i in range(2):
            assert float(cos[p, i]) == pytest.approx(math.cos(p * f[i]) * mag)
            assert float(sin[p, i]) == pytest.approx(math.sin(p * f[i]) * mag)
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0]]], dtype=torch.float64).repeat(4, 1, 1)
    y = plain.rotate_pairs(x, cos[:4], sin[:4], 4)
    assert float(y[3, 0, 0]) == pytest.approx(math.cos(3.0) * mag) and float(y[3, 0, 4]) == 5.0
    assert float(y[3, 0, 2]) == pytest.approx(-2.0 * math.sin(3 * f[1]) * mag)


def test_plain_state_space_by_hand():
    """One head, one row, one column: S <- exp(-A dt) S + dt B x, y = C S + D x."""
    one = lambda *v: torch.tensor(v, dtype=torch.float64)                        # noqa: E731
    xs, B, C, dt = one(1.0, -2.0, 3.0), one(0.5, 1.0, 2.0), one(1.0, 2.0, -1.0), one(0.1, 0.5, 0.2)
    y = plain.state_space(xs.view(3, 1, 1), B.view(3, 1, 1), C.view(3, 1, 1), dt.view(3, 1), one(-2.0), one(0.25))
    S, want = 0.0, []
    for t in range(3):
        S = math.exp(-2.0 * float(dt[t])) * S + float(dt[t] * B[t] * xs[t])
        want.append(float(C[t]) * S + 0.25 * float(xs[t]))
    assert [float(v) for v in y.flatten()] == pytest.approx(want)


def test_plain_gate_comes_before_the_norm_and_groups_are_separate():
    y = torch.tensor([[3.0, 4.0, 1.0, 1.0]], dtype=torch.float64)
    z = torch.full((1, 4), 50.0, dtype=torch.float64)                            # silu(50) = 50 for every channel
    out = plain.gated_group_norm(y, z, torch.tensor([1.0, 2.0, 1.0, 1.0], dtype=torch.float64), 2, 0.0)
    r = math.sqrt(12.5)
    assert out[0].tolist() == pytest.approx([3 / r, 8 / r, 1.0, 1.0])
    z2 = torch.tensor([[50.0, 0.0, 50.0, 50.0]], dtype=torch.float64)            # a closed gate changes its group's norm
    out = plain.gated_group_norm(y, z2, torch.ones(4, dtype=torch.float64), 2, 0.0)
    assert out[0].tolist() == pytest.approx([math.sqrt(2.0), 0.0, 1.0, 1.0])


def test_plain_run_order():
    assert plain.run_order(CFG) == [(0, False)] + [(1, True), (2, False)] * 3 + [(3, False)]
    assert plain.run_order(dict(CFG, loop=None)) == [(i, False) for i in range(4)]
    assert plain.run_order(dict(CFG, loop={"start": 3, "stop": 4, "times": 2})) == \
        [(0, False), (1, False), (2, False), (3, True), (3, True)]

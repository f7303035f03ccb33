"""Rogizen on the GPU against its plain restatement (tests/plain_rogizen.py): each new kernel and part alone, keys at the
chunks' edges with one score made to stand out in every attention kernel, state and convolution inputs that are carried,
freed and taken again, and the engine in float32 and bfloat16 over whole prompts, token-by-token decoding, prompts in pieces
down to two tokens, unequal batches with slots and pages used again, long decoding and greedy generation through the
library's own entry point."""
import json
import os

import pytest
import torch

import helpers
import plain_rogizen as plain
from test_parts_gpu import DEV, DTYPES, build, kernel_plan, make_ctx

pytestmark = pytest.mark.gpu


def _attn(heads, kv, dim, conv, scale, chunk, base, dims, scaling):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "conv": conv, "scale": scale,
            "mask": {"size": chunk} if chunk else None,
            "rot": {"base": base, "dims": dims, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))
                    if scaling else None}}


def _ssm(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


# A: every layer differs; a loop in the middle that runs three times; chunks shorter than a page, a state whose rows are no
# multiple of 8 (the scan in both precisions), as many key heads as query heads without a mask, one tap.
TINY_A = {"architecture": "Rogizen", "vocab": 211, "width": 96, "embedding": {"scale": 3.0}, "logit_softcap": 20.0,
          "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 3}, "layers": [
    {"type": "mamba2", "mixer": _ssm(3, 12, 20, 1, 1, 3), "mlp": _dense(40)},
    {"type": "attention", "mixer": _attn(6, 3, 32, 3, 0.4, 24, 10000.0, 16, (8.0, 64, 16.0, 2.0)), "mlp": None},
    {"type": "mamba2", "mixer": _ssm(6, 24, 16, 3, 2, 4), "mlp": _dense(72)},
    {"type": "attention", "mixer": _attn(4, 4, 20, 1, 0.5, None, 500.0, 20, None), "mlp": _dense(56)}]}
# B: a width that is no multiple of 8, no cap, no loop, an odd head size, one key head, chunks longer than a page and of
# three tokens, more taps than four, odd numbers of heads, one group per head, one state row per group shared by nothing.
TINY_B = {"architecture": "Rogizen", "vocab": 97, "width": 100, "embedding": {"scale": 1.0}, "logit_softcap": None,
          "norm": {"eps": 1e-6}, "loop": None, "layers": [
    {"type": "attention", "mixer": _attn(3, 1, 16, 5, 0.6, 70, 1000.0, 8, None), "mlp": _dense(44)},
    {"type": "mamba2", "mixer": _ssm(5, 20, 36, 5, 5, 1), "mlp": None},
    {"type": "attention", "mixer": _attn(4, 2, 17, 2, 0.5, 3, 50.0, 4, (2.0, 16, 4.0, 1.0)), "mlp": None},
    {"type": "mamba2", "mixer": _ssm(1, 12, 40, 1, 1, 6), "mlp": _dense(28)},
    {"type": "mamba2", "mixer": _ssm(4, 9, 1, 2, 3, 2), "mlp": None}]}
# C: head sizes 64, 128 and 96 (each of the fast attention kernels), chunks of a page + 1, of 100 and of 128, states of 128
# rows, 72 and 24 with narrow heads (the tensor-core scan in its instantiations), a loop at the start followed by layers.
TINY_C = {"architecture": "Rogizen", "vocab": 160, "width": 128, "embedding": {"scale": 0.7}, "logit_softcap": 40.0,
          "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 2}, "layers": [
    {"type": "attention", "mixer": _attn(4, 2, 64, 4, 0.25, 65, 20000.0, 64, (3.0, 128, 16.0, 1.0)), "mlp": _dense(96)},
    {"type": "mamba2", "mixer": _ssm(4, 64, 128, 2, 2, 4), "mlp": None},
    {"type": "attention", "mixer": _attn(2, 1, 128, 4, 0.2, 100, 10000.0, 32, None), "mlp": None},
    {"type": "mamba2", "mixer": _ssm(2, 40, 72, 1, 1, 4), "mlp": _dense(64)},
    {"type": "attention", "mixer": _attn(2, 2, 96, 2, 0.2, 128, 3000.0, 96, (4.0, 32, 8.0, 0.5)), "mlp": None},
    {"type": "mamba2", "mixer": _ssm(8, 16, 24, 4, 8, 2), "mlp": None}]}
CFGS = {"a": TINY_A, "b": TINY_B, "c": TINY_C}
LENGTHS = {"a": [1, 2, 5, 64, 65, 130, 300], "b": [3, 77, 200, 257], "c": [40, 129, 260]}
SHARPEN = {"a": 1.25, "b": 1.2, "c": 1.0}        # factor on the weights of the query norms
_folders, _engines = {}, {}


def folder_for(tag):
    """A model folder of random weights: wide embeddings, sharp attention scores (a few keys carry nearly all the weight,
    so one that is lost or added shows), convolutions whose older taps matter, states that live for many tokens."""
    from llm_infer_engine_b200.weights.random_init import random_tensors
    from llm_infer_engine_b200.weights.safetensors_io import save_file
    if tag not in _folders:
        d = helpers.scratch_folder(f"llmie_rogizen_{tag}_")
        tensors, _ = random_tensors(CFGS[tag], seed=71 + len(_folders), std=0.09, norm_range=(0.7, 1.3))
        g = torch.Generator().manual_seed(9)
        for name in tensors:
            t = tensors[name].float()
            if name == "embed":
                t = t * 8.0
            elif name.endswith((".q.norm", ".k.norm")):
                t = t * SHARPEN[tag]
            elif name.endswith((".conv",)):
                t = torch.rand(t.shape, generator=g) * 1.6 - 0.8
            elif name.endswith(".A_log"):
                t = torch.rand(t.shape, generator=g) * 3.0 - 2.0
            elif name.endswith(".D"):
                t = torch.rand(t.shape, generator=g) + 0.5
            elif name.endswith(("mix.o", ".down")):
                t = t * 2.0
            tensors[name] = t.to(torch.bfloat16)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(CFGS[tag], f)
        save_file(tensors, os.path.join(d, "model.safetensors"))
        _folders[tag] = d
    return _folders[tag]


def plain_weights(tag):
    from safetensors.torch import load_file
    return {k: v.double() for k, v in load_file(os.path.join(folder_for(tag), "model.safetensors")).items()}


def engine_for(tag, dtype, **kw):
    from llm_infer_engine_b200 import Engine
    key = (tag, dtype, tuple(sorted(kw.items())))
    if key not in _engines:
        _engines[key] = Engine(folder_for(tag), dtype=dtype, max_batch=kw.pop("max_batch", 8),
                               max_tokens=kw.pop("max_tokens", 64 * 48), cuda_graph=kw.pop("cuda_graph", False), **kw)
    return _engines[key]


def bound(dtype, want):
    return (3e-5 if dtype == "float32" else 0.05) * max(1.0, float(want.abs().max()))


_oracle = {}


def oracle(tag, requests):
    w = plain_weights(tag)
    out = {}
    for rid, toks in requests.items():
        key = (tag, tuple(toks))
        if key not in _oracle:
            _oracle[key] = plain.forward(CFGS[tag], w, toks).float()
        out[rid] = _oracle[key]
    return out


def compare(got, want, dtype, what):
    for rid in want:
        assert got[rid].shape == want[rid].shape, (what, rid)
        diff = (got[rid] - want[rid]).abs().max(dim=1).values
        tol_ = bound(dtype, want[rid])
        over = int((diff > tol_).sum())
        allowed = 0 if dtype == "float32" else max(1, len(diff) // 50)
        assert over <= allowed and float(diff.max()) <= (tol_ if dtype == "float32" else 2 * tol_), (
            f"{what}: request {rid}: {over} of {len(diff)} positions over the bound {tol_:.3e}, worst "
            f"{float(diff.max()):.3e}, first at token {int((diff > tol_).nonzero()[0])}")


def requests_for(tag):
    return {f"r{i}": helpers.random_tokens(CFGS[tag]["vocab"], n, seed=40 + i) for i, n in enumerate(LENGTHS[tag])}


def tol(dtype, scale):
    return (2e-5 if dtype == "float32" else 2e-2) * max(1.0, scale)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [200, 202, 2048])
def test_add_with_a_bias_norm_and_plain_copy(dtype, size):
    """h += y + b with the norm behind it, with rows, and with the new stream itself stored into columns of a wider row."""
    from llm_infer_engine_b200.parts import ScaledDelta
    norm, w = build("norm", "rmsnorm", {"size": size, "eps": 1e-5, "weight_name": ""}, dtype, seed=2)
    g = torch.Generator().manual_seed(size)
    h, y = torch.randn(7, size, generator=g) * 3, torch.randn(7, size, generator=g)
    b, s = torch.randn(size, generator=g), torch.rand(size, generator=g) + 0.5
    for bias, ref in ((b, h.double() + y.double() + b.double()), (None, h.double() + y.double())):
        delta = ScaledDelta([(y.to(DEV), 1.0)], bias=None if bias is None else bias.to(DEV))
        hd = h.clone().to(DEV)
        x = norm.forward(hd, delta)
        want = plain.rms(ref, 1e-5) * w[""].double()
        assert float((hd.cpu().double() - ref).abs().max()) <= 1e-5
        assert float((x.float().cpu().double() - want).abs().max()) <= tol(dtype, float(want.abs().max()))
        rows = i32([5, 0])
        some = norm.forward(h.to(DEV), delta, rows=rows)
        assert float((some.float().cpu().double() - want[[5, 0]]).abs().max()) <= tol(dtype, float(want.abs().max()))
        wide = torch.full((7, 2 * size), 9.0, dtype=DTYPES[dtype], device=DEV)
        hd = h.clone().to(DEV)
        delta.add_into(hd, wide[:, size:])
        assert float((hd.cpu().double() - ref).abs().max()) <= 1e-5
        assert float((wide[:, size:].float().cpu().double() - ref).abs().max()) <= tol(dtype, float(ref.abs().max()))
        assert float((wide[:, :size].float() - 9.0).abs().max()) == 0.0
    scaled = ScaledDelta.of(ScaledDelta([(y.to(DEV), 2.0)], bias=b.to(DEV)), s.to(DEV)).materialize().cpu().double()
    assert float((scaled - s.double() * (2 * y.double() + b.double())).abs().max()) <= 1e-5
    # a float32 branch output in front of a bfloat16 norm: added by the same kernel
    hd = h.clone().to(DEV)
    norm.forward(hd, y.to(DEV))
    assert float((hd.cpu().double() - (h.double() + y.double())).abs().max()) <= 1e-5


@pytest.mark.parametrize("rows", [1, 3, 8, 16])
def test_product_added_with_a_bias(rows):
    from llm_infer_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(rows)
    x, w = (torch.randn(n, 96, generator=g).to(torch.bfloat16) for n in (rows, 80))
    h, b = torch.randn(rows, 80, generator=g), torch.randn(80, generator=g)
    got = ops.gemm_skinny_add_bias(x.to(DEV), w.to(DEV), h.clone().to(DEV), b.to(DEV)).cpu().double()
    want = h.double() + x.double() @ w.double().T + b.double()
    assert float((got - want).abs().max()) <= 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("channels,taps", [(24, 4), (30, 4), (40, 2), (9, 7), (16, 1), (128, 3)])
def test_convolution_in_pieces_carries_its_inputs(dtype, channels, taps):
    """Pieces down to one token (shorter than the taps), single-token steps that write the state themselves, an activation,
    a bias in front and behind, outputs of both types; another slot's state is left alone."""
    from llm_infer_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(channels + taps)
    lens = [90, 40]
    dt = DTYPES[dtype]
    proj = [torch.randn(n, channels + 8, generator=g).to(dt) for n in lens]
    xb, cb = torch.randn(channels, generator=g), torch.randn(channels, generator=g)
    w = torch.rand(channels, taps, generator=g) - 0.5
    want = [plain.silu(plain.short_conv(p[:, 8:].double() + xb.double(), w.double()) + cb.double()) for p in proj]
    state = torch.zeros(4, taps - 1, channels, device=DEV) if taps > 1 else None
    if taps > 1:
        state[1] = 5.0
    slots = i32([2, 0])
    held = [0, 0]
    for pieces in ([1, 1], [2, 30], [1, 1], [0, 1], [1, 0], [70, 2], [1, 1], [14, 4]):
        live = [i for i in range(2) if pieces[i]]
        cu, tok_seq = [0], []
        for k, i in enumerate(live):
            cu.append(cu[-1] + pieces[i])
            tok_seq += [k] * pieces[i]
        x = torch.cat([proj[i][held[i]:held[i] + pieces[i]] for i in live]).to(DEV)
        single = all(pieces[i] == 1 for i in live)
        out = torch.empty(cu[-1], channels, dtype=dt if sum(held) % 2 else torch.float32, device=DEV)
        ops.causal_conv(x, 8, xb.to(DEV), w.t().contiguous().to(DEV), cb.to(DEV), state, i32(cu), i32(tok_seq), slots[live].contiguous(), out,
                        act=ops.ACT_SILU, single=single)
        if taps > 1 and not single:
            ops.conv_state_store(x, 8, xb.to(DEV), state, i32(cu), slots[live].contiguous(), len(live))
        ref = torch.cat([want[i][held[i]:held[i] + pieces[i]] for i in live])
        limit = 1e-5 if out.dtype == torch.float32 else 2e-2
        assert float((out.float().cpu().double() - ref).abs().max()) <= limit * max(1.0, float(ref.abs().max())), pieces
        held = [h + p for h, p in zip(held, pieces)]
    if taps > 1:
        assert float((state[1] - 5.0).abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0


def _steps(g, n, H, G, N, P):
    """Random inputs of the recurrence: x, B, C, steps of very different sizes, decays from slow to fast."""
    xs, B, C = torch.randn(n, H, P, generator=g), torch.randn(n, G, N, generator=g), torch.randn(n, G, N, generator=g)
    raw = torch.randn(n, H, generator=g) * 2 - 1
    return xs, B / N ** 0.5, C, raw


SHAPES = [(3, 1, 20, 24), (4, 4, 9, 5), (6, 2, 128, 64), (2, 1, 72, 40), (8, 4, 24, 16), (1, 1, 256, 32), (5, 5, 36, 20),
          (2, 2, 8, 8), (3, 3, 300, 12)]


@pytest.mark.parametrize("form", ["scan", "step", "tensor"])
@pytest.mark.parametrize("H,G,N,P", SHAPES)
def test_state_space_recurrence_in_every_form(form, H, G, N, P):
    """The float32 scan (pieces in chunks beside short ones), the one-token kernel and the tensor-core kernel against the
    plain loop, each carrying the state through the slots; a chunk's edge at 64 tokens inside, at and after a piece's end;
    another slot's state is left alone."""
    from llm_infer_engine_b200.kernels import ops
    if form == "tensor" and not ops.ssm_scan_supported(N, P):
        pytest.skip("sizes the tensor-core kernel does not take")
    g = torch.Generator().manual_seed(H * 1000 + N + P)
    dt_b, A, D = torch.randn(H, generator=g), torch.rand(H, generator=g) * 4 + 0.02, torch.randn(H, generator=g)
    lens = [335, 212, 66]
    inner = H * P
    store = torch.bfloat16 if form == "tensor" else torch.float32
    seqs, want = [], []
    for n in lens:
        xs, B, C, raw = _steps(g, n, H, G, N, P)
        xs, B, C = (t.to(store).double() for t in (xs, B, C))
        dt = torch.nn.functional.softplus(raw.double() + dt_b.double())
        want.append(plain.state_space(xs, B, C, dt, -A.double(), D.double()).reshape(n, inner))
        seqs.append((torch.cat([xs.reshape(n, -1), B.reshape(n, -1), C.reshape(n, -1)], dim=1).to(store), raw))
    state = torch.zeros(5, H, N, P, device=DEV)
    state[2] = 7.0
    slots = i32([3, 1, 4])
    held = [0, 0, 0]
    pieces_list = [[1, 1, 1]] * 4 if form == "step" else \
        [[20, 1, 2], [44, 64, 0], [1, 1, 1], [64, 65, 63], [206, 81, 0]]
    for pieces in pieces_list:
        live = [i for i in range(3) if pieces[i]]
        cu = [0]
        for i in live:
            cu.append(cu[-1] + pieces[i])
        xbc = torch.cat([seqs[i][0][held[i]:held[i] + pieces[i]] for i in live]).to(DEV).contiguous()
        raw = torch.cat([seqs[i][1][held[i]:held[i] + pieces[i]] for i in live])
        proj = torch.cat([torch.zeros(cu[-1], 3), raw], dim=1).to(DEV)
        out = torch.empty(cu[-1], inner, device=DEV)
        sl = slots[live].contiguous()
        if form == "scan":
            dt, decay = torch.empty(cu[-1], H, device=DEV), torch.empty(cu[-1], H, device=DEV)
            ops.ssm_steps(proj, 3, dt_b.to(DEV), A.to(DEV), dt, decay)
            ops.matrix_scan(xbc[:, inner + G * N:].contiguous(), xbc[:, inner:inner + G * N].contiguous(), xbc[:, :inner],
                            state, i32(cu), sl, out, len(live), H, N, P, max_len=max(pieces), head_decay=decay,
                            key_factor=dt, groups=G)
            out += (xbc[:, :inner].view(-1, H, P) * D.to(DEV)[:, None]).reshape(-1, inner)
        else:
            fn = ops.ssm_step if form == "step" else ops.ssm_scan
            fn(proj, 3, dt_b.to(DEV), A.to(DEV), D.to(DEV), xbc, state, i32(cu), sl, out, len(live), H, G, N, P)
        ref = torch.cat([want[i][held[i]:held[i] + pieces[i]] for i in live])
        # the tensor-core form keeps what the recurrence makes to 16 bits and more: far below bfloat16's own 8
        limit = 3e-4 if form == "tensor" else 3e-5
        assert float((out.cpu().double() - ref).abs().max()) <= limit * max(1.0, float(ref.abs().max())), pieces
        held = [h + p for h, p in zip(held, pieces)]
    assert float((state[2] - 7.0).abs().max()) == 0.0 and float(state[0].abs().max()) == 0.0


@pytest.mark.parametrize("form", ["step", "tensor"])
def test_a_read_only_step_leaves_the_state(form):
    from llm_infer_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    xbc = torch.randn(2, 2 * 8 + 2 * 8, generator=g).to(torch.bfloat16 if form == "tensor" else torch.float32)
    state = torch.randn(2, 2, 8, 8, generator=g).to(DEV)
    before = state.clone()
    v = torch.ones(2, device=DEV)
    fn = ops.ssm_step if form == "step" else ops.ssm_scan
    fn(torch.zeros(2, 2, device=DEV), 0, v, v, v, xbc.to(DEV), state, i32([0, 1, 2]), i32([1, 0]),
       torch.empty(2, 16, device=DEV), 2, 2, 1, 8, 8, write_state=False)
    assert torch.equal(state, before)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,vdim,groups", [(6, 24, 2), (3, 12, 1), (5, 9, 3), (64, 64, 1), (8, 16, 8), (32, 64, 4)])
def test_gated_norm_in_groups(dtype, heads, vdim, groups):
    """With and without the skip term; z a run of columns of a wider row."""
    from llm_infer_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(heads)
    n = heads * vdim
    y, x = torch.randn(11, n, generator=g) * 3, torch.randn(11, n + 4, generator=g)
    z = (torch.randn(11, n + 16, generator=g) * 2).to(DTYPES[dtype])
    w, D = torch.rand(n, generator=g) + 0.5, torch.randn(heads, generator=g)
    out = torch.empty(11, n, dtype=DTYPES[dtype], device=DEV)
    ops.gated_group_norm(y.to(DEV), z.to(DEV)[:, :n], w.to(DEV), 1e-5, out, groups)
    ref = plain.gated_group_norm(y.double(), z[:, :n].double(), w.double(), groups, 1e-5)
    assert float((out.float().cpu().double() - ref).abs().max()) <= tol(dtype, float(ref.abs().max()))
    ops.gated_group_norm(y.to(DEV), z.to(DEV)[:, :n], w.to(DEV), 1e-5, out, groups, skip_x=x.to(DEV)[:, :n], skip=D.to(DEV))
    full = y.double() + (x[:, :n].double().view(11, heads, vdim) * D.double()[:, None]).reshape(11, n)
    ref = plain.gated_group_norm(full, z[:, :n].double(), w.double(), groups, 1e-5)
    assert float((out.float().cpu().double() - ref).abs().max()) <= tol(dtype, float(ref.abs().max()))


# ------------------------------------------------------------------------------------------ parts alone
def _run_mixer_in_pieces(mixer, cache, dtype, xs, want, schedule, factor=2.0):
    slots = [cache.take_slot() for _ in xs]
    held = [0] * len(xs)
    for pieces in schedule:
        live = [i for i, p in enumerate(pieces) if p > 0]
        for i in live:
            cache.reserve(slots[i], held[i] + pieces[i])
        ctx = make_ctx([pieces[i] for i in live], [held[i] for i in live], [slots[i] for i in live], dtype,
                       kernels=kernel_plan(dtype))
        x = torch.cat([xs[i][held[i]:held[i] + pieces[i]] for i in live])
        y = mixer.forward(x.to(DEV), ctx, cache.unit(0), True).materialize().cpu().double()
        ref = torch.cat([want[i][held[i]:held[i] + pieces[i]] for i in live])
        assert float((y - ref).abs().max()) <= tol(dtype, float(ref.abs().max())) * factor, (pieces, held)
        for i in live:
            held[i] += pieces[i]
            cache.note_appended(slots[i], held[i], device_updated=False)
    return slots


PIECES = ([1, 2], [99, 28], [39, 2], [1, 1], [1, 1], [0, 34])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag,layer", [("a", 1), ("a", 3), ("b", 0), ("b", 2), ("c", 0), ("c", 2), ("c", 4)])
def test_attention_behind_a_convolution(dtype, tag, layer):
    """Two sequences over prompts in pieces and single tokens, then a slot given back and taken again, whose convolution
    must start from zeros."""
    from llm_infer_engine_b200.cache import Cache
    cfg = CFGS[tag]
    m = cfg["layers"][layer]["mixer"]
    mixer, w = build("mixer", "conv_attention", {
        "hidden": cfg["width"], "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"], "taps": m["conv"],
        "scale": m["scale"], "norm_eps": 1e-5, "chunk": m["mask"]["size"] if m["mask"] else 0,
        "rot_dims": m["rot"]["dims"], "rot_base": m["rot"]["base"], "rot_scaling": m["rot"]["scaling"]}, dtype,
        seed=layer + 3, std=0.25)
    wd = {k: v.double() for k, v in w.items()}
    cache = Cache([mixer.cache_requests()], 3, 64 * 12, 512, DTYPES[dtype], DEV)
    cache.take_slot()
    g = torch.Generator().manual_seed(11)
    xs = [torch.randn(n, cfg["width"], generator=g).to(DTYPES[dtype]) for n in (141, 68)]
    want = [plain.attention(x.double(), m, wd, "", 1e-5) for x in xs]
    slots = _run_mixer_in_pieces(mixer, cache, dtype, xs, want, PIECES)
    cache.give_back_slot(slots[1])
    xs2 = [torch.randn(70, cfg["width"], generator=g).to(DTYPES[dtype])]
    _run_mixer_in_pieces(mixer, cache, dtype, xs2, [plain.attention(xs2[0].double(), m, wd, "", 1e-5)], ([2], [67], [1]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag,layer", [("a", 0), ("a", 2), ("b", 1), ("b", 3), ("b", 4), ("c", 1), ("c", 3), ("c", 5)])
def test_state_space_layer(dtype, tag, layer):
    """State and convolution inputs carried through pieces and single tokens; a slot given back and taken again starts
    from zeros."""
    from llm_infer_engine_b200.cache import Cache
    cfg = CFGS[tag]
    m = cfg["layers"][layer]["mixer"]
    mixer, w = build("mixer", "state_space", {
        "hidden": cfg["width"], "n_heads": m["heads"], "v_dim": m["vdim"], "state": m["state"], "groups": m["groups"],
        "norm_groups": m["norm_groups"], "taps": m["conv"], "norm_eps": 1e-5}, dtype, seed=layer + 1, std=0.2)
    w["A_log"] = w["A_log"] * 2 - 2.5                       # decays from slow to fast
    w["dt_bias"] = w["dt_bias"] - 2.0
    mixer.load({k: v.to(DEV, DTYPES[dtype]) for k, v in w.items()})
    wd = {k: v.to(DTYPES[dtype]).double() for k, v in w.items()}
    cache = Cache([mixer.cache_requests()], 3, 64 * 12, 512, DTYPES[dtype], DEV)
    cache.take_slot()
    g = torch.Generator().manual_seed(13)
    xs = [torch.randn(n, cfg["width"], generator=g).to(DTYPES[dtype]) for n in (300, 68)]
    want = [plain.mamba2(x.double(), m, wd, "", 1e-5) for x in xs]
    slots = _run_mixer_in_pieces(mixer, cache, dtype, xs, want, ([130, 30], [1, 2], [1, 1], [168, 35]), factor=4.0)
    cache.give_back_slot(slots[0])
    xs2 = [torch.randn(30, cfg["width"], generator=g).to(DTYPES[dtype])]
    _run_mixer_in_pieces(mixer, cache, dtype, xs2, [plain.mamba2(xs2[0].double(), m, wd, "", 1e-5)], ([1], [1], [3], [25]),
                         factor=4.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["none", "tensor", "delta"])
def test_embedding_mixed_into_the_stream(dtype, kind):
    """h <- Win [h + pending; x0] twice in one step: the second pass sees the new stream and the SAME x0."""
    from llm_infer_engine_b200.parts import ScaledDelta
    stage, w = build("stream", "embedding_mix", {"size": 96}, dtype, seed=5)
    g = torch.Generator().manual_seed(6)
    x0, y, b = torch.randn(9, 96, generator=g), torch.randn(9, 96, generator=g), torch.randn(96, generator=g)
    ctx = make_ctx([9], [0], [0], dtype)
    h = x0.clone().to(DEV)
    stage.begin(h, ctx)
    pending = {"none": None, "tensor": y.to(DEV), "delta": ScaledDelta([(y.to(DEV), 1.0)], bias=b.to(DEV))}[kind]
    extra = {"none": 0, "tensor": y.double(), "delta": y.double() + b.double()}[kind]
    h, p = stage.forward(h, pending, ctx)
    W = w["in"].double()
    want = torch.cat([x0.double() + extra, x0.double()], dim=1) @ W.T
    assert p is None and h.dtype == torch.float32
    assert float((h.cpu().double() - want).abs().max()) <= tol(dtype, float(want.abs().max()))
    h2, _ = stage.forward(h, None, ctx)
    want2 = torch.cat([h.cpu().double(), x0.double()], dim=1) @ W.T
    assert float((h2.cpu().double() - want2).abs().max()) <= tol(dtype, float(want2.abs().max()))


# ------------------------------------------------------------------------------------------ the chunks' edges
def _chunk_edge_case(dtype, hd, n_q, n_kv, chunk, n, q_len, probe):
    """Attention in chunks: a sequence of n rows of which the last q_len are this step's queries; the LAST query points
    straight at row `probe`, whose value is a marker (20 in every entry). Slots and pages were given back and taken again
    before, so the sequence's pages are out of order."""
    from llm_infer_engine_b200.cache import Cache, KVRequest
    from llm_infer_engine_b200.parts import AttentionOptions
    cache = Cache([[KVRequest(n_kv, hd, chunk=chunk)]], 4, 64 * 24, 1024, DTYPES[dtype], DEV)
    cache.take_slot()
    other = cache.take_slot()
    cache.reserve(other, 130)
    slot = cache.take_slot()
    cache.reserve(slot, 70)
    cache.give_back_slot(other)
    cache.reserve(slot, n)
    g = torch.Generator().manual_seed(n * 7 + probe)
    k, v = torch.randn(n, n_kv, hd, generator=g) * 0.1, torch.randn(n, n_kv, hd, generator=g) * 0.1
    q = torch.randn(q_len, n_q, hd, generator=g) * 0.1
    k[probe], v[probe], q[-1] = 2.0, 20.0, 2.0
    k, v, q = (t.to(DTYPES[dtype]) for t in (k, v, q))
    kv = cache.unit(0).kv
    table = kv.block_table[slot].cpu()
    for j in range(n):
        kv.k[int(table[j // 64]), :, j % 64] = k[j].to(DEV)
        kv.v[int(table[j // 64]), :, j % 64] = v[j].to(DEV)
    ctx = make_ctx([q_len], [n - q_len], [slot], dtype, kernels=kernel_plan(dtype))
    out = torch.empty(q_len, n_q * hd, dtype=DTYPES[dtype], device=DEV)
    ctx.attention(q.reshape(q_len, -1).to(DEV), kv, out, n_q, n_kv, hd, AttentionOptions(scale=1.0, chunk=chunk))
    ok = plain.same_chunk_mask(n, chunk)[n - q_len:]
    kk, vv = (t.double().repeat_interleave(n_q // n_kv, dim=1) for t in (k, v))
    s = torch.einsum("ihd,jhd->hij", q.double(), kk).masked_fill(~ok, float("-inf"))
    want = torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), vv).reshape(q_len, -1)
    return out.float().cpu(), want.float(), bool(ok[-1, probe])


EDGES = [  # chunk, keys, probe, may the last query (position keys - 1) see it
    (80, 300, 240, True), (80, 300, 239, False),          # just inside and just outside an edge inside a page
    (64, 257, 256, True), (64, 257, 255, False),          # a chunk that begins with the last query, on a page's edge
    (64, 256, 192, True), (64, 256, 191, False),          # a chunk of exactly one page
    (65, 260, 195, True), (65, 260, 194, False), (65, 261, 194, False),
    (128, 500, 384, True), (128, 500, 383, False), (128, 640, 512, True), (128, 640, 511, False),
    (300, 299, 0, True), (300, 700, 600, True), (300, 700, 599, False), (1000, 700, 0, True),   # keys far back
    (1, 40, 39, True), (1, 40, 38, False), (2, 130, 128, True), (2, 130, 127, False), (3, 131, 129, True),
    (3, 131, 128, False), (1, 1, 0, True), (7, 2, 0, True)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hd,n_q,n_kv", [(64, 4, 2), (128, 2, 1), (96, 3, 1), (32, 4, 4), (20, 2, 2)])
@pytest.mark.parametrize("q_len", [1, 2, 37, 260])
def test_keys_at_every_edge_of_a_chunk_stand_out(dtype, hd, n_q, n_kv, q_len):
    """A probe row that the query may see puts the marker into the output (about 20); one that it may not see leaves the
    output small. Plain kernel (float32, odd sizes), tcgen05 prompts and their one-token kernel (64, 128), the kernel by
    rows (96, prompts of 32), the split kernel (one token at 32); every other query of the step is checked too."""
    for chunk, n, probe, visible in EDGES:
        if q_len > n:
            continue
        got, want, ok = _chunk_edge_case(dtype, hd, n_q, n_kv, chunk, n, q_len, probe)
        assert ok == visible
        assert float((got - want).abs().max()) <= (1e-3 if dtype == "float32" else 0.3), (chunk, n, probe)
        assert (float(got[-1].abs().max()) > 10) == visible, (chunk, n, probe, float(got[-1].abs().max()))
    if dtype == "bfloat16":
        from llm_infer_engine_b200.kernels import ops
        ops.check_tc_status("cuda")


# ------------------------------------------------------------------------------------------ the engine
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["a", "b", "c"])
def test_every_schedule_matches_plain(tag, dtype):
    """Whole prompts; the last tokens one by one (more of them than the longest chunk); unequal batches in which shorter
    requests end early and the next batch takes their slots, pages and state; prompts in pieces of 2, 7, 64 and 100 tokens;
    a prompt in pieces beside sequences that go on by one token."""
    requests = requests_for(tag)
    want = oracle(tag, requests)
    engine = engine_for(tag, dtype)
    plans = {"whole": helpers.plan_whole(requests), "tail": helpers.plan_tail(requests, 140),
             "batched": helpers.plan_batched(requests, 3, 0.6), "mixed": helpers.plan_mixed(requests, 9)}
    some = {rid: toks for rid, toks in requests.items() if len(toks) <= 200}
    for chunk in (2, 7, 64, 100):
        plans[f"pieces of {chunk}"] = helpers.plan_chunked(some if chunk == 2 else requests, chunk)
    for name, steps in plans.items():
        got = helpers.run_plan_engine(engine, steps)
        compare(got, {rid: want[rid] for rid in got}, dtype, f"{tag}/{dtype}/{name}")
        assert engine.cache.free_slots() == engine.cache.n_slots and engine.cache.free_pages() == engine.cache.n_pages
    if dtype == "bfloat16":
        from llm_infer_engine_b200.kernels import ops
        ops.check_tc_status("cuda")


def test_the_models_are_sharp_enough_to_show_what_a_fault_would_change():
    """The bounds above mean something only if a fault moves the logits by more than they allow. In the plain
    implementation: a chunk one token off, no chunks at all, the convolution's older taps lost, the rotation's scaling left
    out, values after the norm instead of before it, states or convolution inputs that are lost at a position, the skip
    term and the biases left out, the gate after the norm, one norm group instead of several, a pass of the loop left out,
    and the embedding left out of the loop's projection each differ by several bounds."""
    def rms_then_gate(y, z, weight, groups, eps):
        n = y.shape[1]
        return plain.rms(y.view(len(y), groups, n // groups), eps).reshape(len(y), n) * plain.silu(z) * weight

    for tag in ("a", "b", "c"):
        w, cfg = plain_weights(tag), CFGS[tag]
        toks = helpers.random_tokens(cfg["vocab"], 200, seed=47)
        right = plain.forward(cfg, w, toks)

        def gap(what, cfg2=cfg, w2=w, **patched):
            saved = {k: getattr(plain, k) for k in patched}
            try:
                for k, v in patched.items():
                    setattr(plain, k, v)
                diff = (plain.forward(cfg2, w2, toks) - right).abs().max(dim=1).values
            finally:
                for k, v in saved.items():
                    setattr(plain, k, v)
            tol_ = bound("bfloat16", right)
            over = int((diff > tol_).sum())
            assert over > max(1, len(diff) // 50) and float(diff.max()) > 2 * tol_, (tag, what, over, float(diff.max()), tol_)

        def changed(fn):
            c = json.loads(json.dumps(cfg))
            fn(c)
            return c

        def chunk_off(c):
            for layer in c["layers"]:
                if layer["type"] == "attention" and layer["mixer"]["mask"]:
                    layer["mixer"]["mask"]["size"] += 1

        def no_mask(c):
            for layer in c["layers"]:
                if layer["type"] == "attention":
                    layer["mixer"]["mask"] = None

        def no_scaling(c):
            for layer in c["layers"]:
                if layer["type"] == "attention":
                    layer["mixer"]["rot"]["scaling"] = None

        def one_group(c):
            for layer in c["layers"]:
                if layer["type"] == "mamba2":
                    layer["mixer"]["norm_groups"] = 1

        right_conv, right_ssm = plain.short_conv, plain.state_space

        def lost_inputs(u, taps):                        # the convolution starts anew at position 100
            return torch.cat([right_conv(u[:100], taps), right_conv(u[100:], taps)])

        def lost_state(xs, B, C, dt, A, D):
            return torch.cat([right_ssm(*(t[:100] for t in (xs, B, C, dt)), A, D),
                              right_ssm(*(t[100:] for t in (xs, B, C, dt)), A, D)])

        gap("chunk one off", changed(chunk_off))
        gap("no chunks", changed(no_mask))
        gap("last tap only", short_conv=lambda u, taps: u * taps[:, -1])
        gap("lost inputs", short_conv=lost_inputs)
        gap("lost state", state_space=lost_state)
        gap("gate after norm", gated_group_norm=rms_then_gate)
        gap("one norm group", changed(one_group))
        if tag != "b":                                   # there the only scaled layer sees three tokens at most
            gap("no scaling", changed(no_scaling))
        gap("no skip", w2={k: (v * 0 if k.endswith(".D") else v) for k, v in w.items()})
        gap("no biases", w2={k: (v * 0 if k.endswith((".q.b", ".k.b", ".o.b")) else v) for k, v in w.items()})
        if cfg["loop"]:
            gap("a pass missing", dict(cfg, loop=dict(cfg["loop"], times=cfg["loop"]["times"] - 1)))
            d = cfg["width"]
            gap("no embedding", w2=dict(w, **{"loop.in": torch.cat([w["loop.in"][:, :d], w["loop.in"][:, d:] * 0], dim=1)}))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batch_and_cutting_do_not_change_a_row(dtype):
    """The logits of a position do not depend on what else is in the batch or how the prompt was cut: float32 kernels sum
    in a fixed order, so there the rows are equal bit for bit."""
    tag = "a"
    requests = requests_for(tag)
    engine = engine_for(tag, dtype)
    alone = helpers.run_plan_engine(engine, helpers.plan_whole(requests))
    together = helpers.run_plan_engine(engine, helpers.plan_batched(requests, 8, 1.0))
    pieces = helpers.run_plan_engine(engine, helpers.plan_chunked(requests, 7))
    for rid in requests:
        if dtype == "float32":
            if len(requests[rid]) > 1:                   # a lone single token is a one-token step: another kernel
                assert torch.equal(alone[rid], together[rid]), rid
            assert float((alone[rid] - pieces[rid]).abs().max()) <= 0.3 * bound(dtype, alone[rid]), rid
        else:
            # other kernels serve other batch sizes, so roundings differ, and sharp attention carries a difference on
            compare({rid: together[rid]}, {rid: alone[rid]}, dtype, "together against alone")


def test_trace_run_program_and_other_sizes_at_once(tmp_path):
    """bin/trace_run as a subprocess on the configuration with the odd sizes."""
    tag = "b"
    requests = {k: v for k, v in requests_for(tag).items() if len(v) <= 200}
    want = oracle(tag, requests)
    steps = helpers.plan_batched(requests, 4, 0.5)
    peak = max(sum(len(v) for v in requests.values()), 64)
    for dtype in ("float32", "bfloat16"):
        got = helpers.run_plan_trace_run(folder_for(tag), dtype, steps, peak, CFGS[tag]["vocab"])
        compare(got, want, dtype, f"trace_run/{dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_prompt_length_that_comes_again_is_replayed_right(dtype):
    """Lone prompts of one length run eagerly, are captured, and are replayed, in other slots and at other start positions:
    the convolution's inputs, the states, the loop's projection and the chunks inside the captured step."""
    tag = "c"
    engine = engine_for(tag, dtype, cuda_graph=True)
    toks = [helpers.random_tokens(CFGS[tag]["vocab"], 90, seed=90 + i) for i in range(3)]
    want = oracle(tag, {str(i): t for i, t in enumerate(toks)})
    held = [engine.open() for _ in range(2)]                 # so that the slots differ from call to call
    for i, t in enumerate(toks):
        slot = engine.open()
        for lo in (0, 30, 60):                               # three pieces of one length
            got = engine.step([slot], [t[lo:lo + 30]], "last").float().cpu()[0]
            ref = want[str(i)][lo + 29]
            assert float((got - ref).abs().max()) <= bound(dtype, want[str(i)]), (i, lo)
        if i == 0:
            engine.close(held.pop())
        engine.close(slot)
    assert any(g for g in engine._prefill_graphs.values())
    engine.close(held.pop())


@pytest.mark.parametrize("dtype,gap", [("float32", 1e-4), ("bfloat16", 0.3)])
@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation_through_the_library(dtype, gap, graph):
    """generate(): admission, ragged prompts, captured one-token steps, slots and their state used again. Greedy tokens
    equal the plain implementation's; where they part the two candidates are a near-tie in the plain logits."""
    from llm_infer_engine_b200 import GenerationStats, generate
    tag = "a"
    w, cfg = plain_weights(tag), CFGS[tag]
    prompts = [helpers.random_tokens(cfg["vocab"], n, seed=60 + i) for i, n in enumerate([1, 5, 42, 64, 3, 90, 2])]
    engine = engine_for(tag, dtype, max_batch=3, max_tokens=64 * 12, cuda_graph=graph)
    stats = GenerationStats()
    out = generate(engine, prompts, max_new_tokens=40, stop_ids=[], stats=stats)          # decoding crosses chunks
    assert stats.batches >= 3 and [len(o) for o in out] == [40] * len(prompts)
    for p, o in zip(prompts, out):
        rows = plain.forward(cfg, w, (p + o)[:-1])[len(p) - 1:]
        for i, tok in enumerate(o):
            best = int(rows[i].argmax())
            assert tok == best or float(rows[i][best] - rows[i][tok]) < gap, (len(p), i, tok, best)
    engine.cache.check()
    assert engine.cache.free_slots() == 3 and engine.cache.free_pages() == engine.cache.n_pages


def test_long_decoding_in_float32():
    """A few hundred captured one-token steps against one whole-sequence pass: the chunks pass over decoded tokens many
    times, their pages are given back and used again, and every state is carried through every step."""
    from llm_infer_engine_b200 import generate
    tag = "b"
    w, cfg = plain_weights(tag), CFGS[tag]
    prompt = helpers.random_tokens(cfg["vocab"], 4, seed=70)
    engine = engine_for(tag, "float32", max_batch=2, max_tokens=64 * 12, cuda_graph=True)
    out = generate(engine, [prompt, prompt[:1]], max_new_tokens=260, stop_ids=[])
    for p, o in zip([prompt, prompt[:1]], out):
        ref = plain.forward(cfg, w, (p + o)[:-1])[len(p) - 1:]
        for i, tok in enumerate(o):
            best = int(ref[i].argmax())
            if tok != best:
                assert float(ref[i][best] - ref[i][tok]) < 1e-4, (i, tok, best)


def test_command_line_generates_with_this_design(tmp_path):
    import subprocess
    import sys
    tag = "c"
    w, cfg = plain_weights(tag), CFGS[tag]
    prompt = helpers.random_tokens(cfg["vocab"], 9, seed=80)
    proc = subprocess.run([sys.executable, os.path.join(helpers.ROOT, "main.py"), "--model", folder_for(tag),
                           "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-new-tokens", "6",
                           "--temperature", "0", "--env-file", str(tmp_path / "none")],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    ids = [int(x) for x in proc.stdout.split("OUTPUT")[1].split("=" * 70)[1].split()]
    seq = list(prompt)
    for tok in ids:
        row = plain.forward(cfg, w, seq)[-1]
        assert tok == int(row.argmax()) or float(row.max() - row[tok]) < 1e-4
        seq.append(tok)
    assert len(ids) == 6

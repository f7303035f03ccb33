"""Selinex on the GPU against its plain restatement (tests/plain_selinex.py): each new kernel and part alone, the
attention's edges with one score made to stand out, states that are carried, freed and taken again, and the engine in
float32 and bfloat16 over whole prompts, token-by-token decoding, prompts in pieces down to two tokens, unequal batches
with slots and pages used again, long decoding and greedy generation through the library's own entry point."""
import json
import os

import pytest
import torch

import helpers
import plain_selinex as plain
from test_parts_gpu import DEV, DTYPES, build, kernel_plan, make_ctx

pytestmark = pytest.mark.gpu


def _left(heads, kv, dim, vdim, window, scale, rot=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window} if window else None}
    return dict(m, rot={"base": rot[0], "dims": rot[1]}) if rot else m


def _moe(experts, count, keep, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}},
            "expert": {"ff": ff}}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _delta(heads, kv, dim, vdim, taps):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": taps}


# A: every layer differs. A loop in the middle; q and k heads that three heads of the state share and one each; a
# convolution of four taps and of one; value heads narrower and wider than key heads; a rotation over a part of a head; no
# mask; a layer without a feed-forward; groups of three experts and of one.
TINY_A = {"architecture": "Selinex", "vocab": 211, "width": 96, "norm": {"eps": 2e-5}, "residual_mult": 0.45,
          "loop": {"start": 1, "stop": 3, "times": 2}, "layers": [
    {"type": "delta", "mixer": _delta(6, 2, 20, 24, 4), "mlp": _moe(12, 4, 2, 3, 40)},
    {"type": "parallel", "mixer": {"left": _left(6, 3, 32, 16, 24, 0.2), "right": {"heads": 3, "dim": 20, "vdim": 24, "tau": 8.0},
                                   "left_scale": 0.7, "right_scale": 1.3}, "mlp": _dense(136, 1.5)},
    {"type": "parallel_2", "mixer": {"left": _left(4, 4, 20, 28, 0, 0.3, (300.0, 12)), "right": {"heads": 2, "dim": 36}},
     "mlp": None},
    {"type": "delta", "mixer": _delta(2, 2, 40, 16, 1), "mlp": _moe(6, 6, 3, 2, 24)}]}
# B: no loop, a width that is no multiple of 8, one key head, a window longer than a page and one of three tokens, heads of
# the state whose rows are more than a warp's lanes take, sizes that are no multiples of 4, one group whose experts are
# all used, a decay without a root.
TINY_B = {"architecture": "Selinex", "vocab": 97, "width": 100, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "loop": None,
          "layers": [
    {"type": "parallel_2", "mixer": {"left": _left(4, 1, 16, 16, 70, 0.25, (500.0, 8)), "right": {"heads": 5, "dim": 12}},
     "mlp": _dense(60, 0.5)},
    {"type": "parallel", "mixer": {"left": _left(2, 2, 24, 8, 3, 0.2), "right": {"heads": 1, "dim": 130, "vdim": 20, "tau": 1.0},
                                   "left_scale": 1.0, "right_scale": 0.25}, "mlp": _moe(5, 1, 1, 5, 20)},
    {"type": "delta", "mixer": _delta(3, 1, 9, 10, 3), "mlp": None}]}
# C: head sizes 64 and 128 with equal value sizes (what the fastest attention kernels take), wide states, a loop at the
# start that runs three times.
TINY_C = {"architecture": "Selinex", "vocab": 160, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 0.6,
          "loop": {"start": 0, "stop": 2, "times": 3}, "layers": [
    {"type": "parallel", "mixer": {"left": _left(4, 2, 64, 64, 100, 0.125), "right": {"heads": 2, "dim": 64, "vdim": 64, "tau": 16.0},
                                   "left_scale": 0.8, "right_scale": 0.6}, "mlp": _dense(256, 1.0)},
    {"type": "parallel_2", "mixer": {"left": _left(2, 1, 128, 128, 65, 0.09, (100000.0, 32)), "right": {"heads": 3, "dim": 64}},
     "mlp": _moe(8, 2, 1, 2, 64)},
    {"type": "delta", "mixer": _delta(4, 2, 128, 64, 4), "mlp": _dense(128, 2.0)}]}
# routed: A once more with routers whose choice changes from token to token (A's leans on the corrections: a choice that
# bfloat16 rounding turns at one token lives on in the states of all later ones, so such a model is for float32).
CFGS = {"a": TINY_A, "b": TINY_B, "c": TINY_C, "routed": TINY_A}
LENGTHS = {"a": [1, 5, 64, 65, 130, 300], "b": [3, 77, 200, 257], "c": [40, 129, 260], "routed": [1, 5, 64, 65, 130, 300]}
SHARPEN = {"a": 3.0, "b": 3.0, "c": 2.0, "routed": 3.0}        # factor on the attention's query and key projections
RANKS = {"a1": 7, "w1": 11}                     # rows of the low-rank products, which a checkpoint decides
_folders, _engines = {}, {}


def folder_for(tag):
    """A model folder of random weights: wide embeddings, sharp attention scores (a few keys carry most of the weight, so
    one that is lost or added shows), corrections that change the router's choice, states that live long, low-rank
    products of ranks that no tile has."""
    from llm_infer_engine_b200.weights.random_init import random_tensors
    from llm_infer_engine_b200.weights.safetensors_io import save_file
    if tag not in _folders:
        d = helpers.scratch_folder(f"llmie_selinex_{tag}_")
        tensors, _ = random_tensors(CFGS[tag], seed=31 + len(_folders), std=0.09, norm_range=(0.5, 1.5))
        g = torch.Generator().manual_seed(6)
        for name in list(tensors):
            t = tensors[name].float()
            last = name.split(".")[-1]
            if name == "embed":
                t = t * 8.0
            elif name.endswith((".left.q", ".left.k")):
                t = t * SHARPEN[tag]
            elif last in ("a1", "w1"):
                t = t[:RANKS[last]]
            elif last in ("a2", "w2"):
                t = t[:, :RANKS["a1" if last == "a2" else "w1"]] * 4.0
            elif last == "correction":
                n = t.shape[0]
                t = torch.randn(n, generator=g) * 0.3 if tag == "routed" else \
                    torch.tensor([0.37 * (e * 5 % n) - 1.5 for e in range(n)])
            elif last == "router":
                t = t * (1.5 if tag == "routed" else 0.3)
            elif last == "norm" and ".mix." in name:
                t = torch.rand(t.shape, generator=g) * 1.9 + 0.05
            elif name.endswith(".a2.b"):
                t = torch.rand(t.shape, generator=g) * 4 - 1
            elif last == "w0":
                t = torch.rand(t.shape, generator=g) * 6 - 6         # fast and slow channels
            elif last == "dt_bias":
                t = torch.rand(t.shape, generator=g) * 3 - 5         # long memories: a state that is lost shows
            elif last == "A_log":
                t = torch.rand(t.shape, generator=g) * 1.5 - 1
            elif last in ("gate", "up") and ".e" not in name:
                t = t * 1.5
            tensors[name] = t.to(torch.bfloat16).contiguous()
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


CLOSE_CALL = 0.02          # a router's choice margin below this may fall the other way in bfloat16
_close_calls, _oracles = {}, {}


def oracle(tag, requests):
    """The plain logits of every request. Beside them it notes, per request, the tokens from the first one on at which
    some router of the plain model chooses by a margin that bfloat16 rounding can turn (the states carry such a choice
    on; the comparison in bfloat16 leaves those tokens out, and sees to it that they are few)."""
    w = plain_weights(tag)
    out = {}
    for rid, toks in requests.items():
        key = (tag, tuple(toks))
        if key not in _oracles:
            margins = []
            logits = plain.forward(w, CFGS[tag], toks, margins_out=margins).float()
            close = torch.zeros(len(toks), dtype=torch.bool)
            for m in margins:
                close |= m < CLOSE_CALL
            close = close.cumsum(0) > 0
            _oracles[key] = (logits, close)
        out[rid], _close_calls[(tag, rid)] = _oracles[key]
    return out


def compare(got, want, dtype, what, tag=None):
    for rid in want:
        assert got[rid].shape == want[rid].shape, (what, rid)
        diff = (got[rid] - want[rid]).abs().max(dim=1).values
        tol_ = bound(dtype, want[rid])
        if dtype != "float32":
            firm = ~_close_calls[(tag, rid)][:len(diff)]
            assert int(firm.sum()) >= 0.7 * len(diff), (what, rid)
            diff = diff[firm]
        over = int((diff > tol_).sum())
        allowed = 0 if dtype == "float32" else max(1, len(diff) // 25)
        worst = float(diff.max())
        assert over <= allowed and worst <= (tol_ if dtype == "float32" else 3 * tol_), (
            f"{what}: request {rid}: {over} of {len(diff)} positions over the bound {tol_:.3e}, worst "
            f"{worst:.3e}, first at token {int((diff > tol_).nonzero()[0])}")


def requests_for(tag):
    return {f"r{i}": helpers.random_tokens(CFGS[tag]["vocab"], n, seed=40 + i) for i, n in enumerate(LENGTHS[tag])}


def tol(dtype, scale):
    return (2e-5 if dtype == "float32" else 2e-2) * max(1.0, scale)


# ------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [202, 204, 2048, 2560, 8192])
@pytest.mark.parametrize("terms,normed", [(1, False), (2, False), (2, True)])
def test_a_branch_closes_and_the_next_opens_in_one_kernel(dtype, size, terms, normed):
    """h += c N(b) (1 + w1) with b one or two terms, each as it is or normed, then N(h) (1 + w2); all rows, selected rows,
    the add alone, and the new stream itself: forms of four channels a thread and element by element."""
    from llm_infer_engine_b200.kernels import ops
    from llm_infer_engine_b200.parts import ScaledDelta
    g = torch.Generator().manual_seed(size + terms)
    around_zero = lambda: (torch.randn(size, generator=g) * 0.3).to(torch.bfloat16).float()           # noqa: E731
    base = {"size": size, "eps": 1e-5, "weight_name": "", "weight_offset": 1.0}
    norm, _ = build("norm", "rmsnorm", base, dtype)
    behind, _ = build("norm", "rmsnorm", dict(base, output_scale=0.35), dtype)
    w_in, w_out = around_zero(), around_zero()
    norm.load({"": w_in.to(DEV)})
    behind.load({"": w_out.to(DEV)})
    h = torch.randn(9, size, generator=g) * 3
    ts = [torch.randn(9, size, generator=g) * s for s in (0.02, 40.0)[:terms]]
    if dtype == "bfloat16":
        ts[-1] = ts[-1].to(torch.bfloat16)                            # terms may be of either type
    cs = (0.5, 0.5) if normed else (0.7, -0.01)
    tw = [torch.rand(size, generator=g) + 0.5 for _ in ts]
    b = sum(c * (plain.rms_unit(t.double(), 1e-5) * v.double() if normed else t.double()) for c, t, v in zip(cs, ts, tw))
    want_h = h.double() + 0.35 * plain.norm_around_one(b, w_out.double(), 1e-5)
    want = plain.norm_around_one(want_h, w_in.double(), 1e-5)
    pair = ScaledDelta([(t.to(DEV), c) for t, c in zip(ts, cs)],
                       term_norms=([v.to(DEV) for v in tw], 1e-5) if normed else None)
    delta = ScaledDelta.normed(pair if terms > 1 or cs[0] != 1.0 else ts[0].to(DEV), behind.weight, behind.eps)
    hd = h.to(DEV)
    rows = torch.tensor([7, 0, 3], dtype=torch.int32, device=DEV)
    y_rows = norm.forward(hd, delta, rows=rows).float().cpu().double()
    assert torch.equal(hd.cpu(), h)                                   # selected rows leave the stream alone
    added = delta.materialize().cpu().double()
    new = torch.empty(9, size, device=DEV)
    ops.sandwich_add_norm(hd.clone(), delta.terms, *(delta.term_norms or ((None, None), 0.0)), *delta.out_norm, None, 0.0, new)
    y = norm.forward(hd, delta).float().cpu().double()
    assert float((hd.cpu().double() - want_h).abs().max()) <= 2e-5
    assert float((new.cpu().double() - want_h).abs().max()) <= 2e-5
    assert float((added - (want_h - h.double())).abs().max()) <= 2e-5
    assert float((y - want).abs().max()) <= tol(dtype, float(want.abs().max()))
    assert float((y_rows - want[[7, 0, 3]]).abs().max()) <= tol(dtype, float(want.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens,ff,limit", [(1, 64, 0.4), (5, 136, 1.25), (40, 100, 0.8), (300, 64, 3.0)])
def test_feed_forward_with_a_clamped_gate(dtype, tokens, ff, limit):
    """Gates far below and beyond the limit, linear parts on both sides of it; the skinny product's form and the other."""
    part, w = build("feed_forward", "swiglu", {"hidden": 64, "intermediate": ff, "activation": "clamped", "gate_alpha": 1.702,
                                               "gate_limit": limit, "out_float32": True,
                                               "names": {"gate": "gate", "up": "up", "down": "down"}}, dtype, seed=ff, std=0.3)
    x = torch.randn(tokens, 64, generator=torch.Generator().manual_seed(tokens)).to(DTYPES[dtype])
    y = part.forward(x.to(DEV), make_ctx([tokens], [0], [0], dtype)).float().cpu().double()
    wd = {k: v.double() for k, v in w.items()}
    want = plain.dense_ff(x.double(), wd, "", {"limit": limit})
    assert float((y - want).abs().max()) <= tol(dtype, float(want.abs().max())) * 2
    for other in (limit * 2, limit / 2):
        assert float((plain.dense_ff(x.double(), wd, "", {"limit": other}) - want).abs().max()) > 0.1 * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,count,keep,top,ff", [(12, 4, 2, 3, 40), (6, 6, 3, 2, 24), (5, 1, 1, 5, 20), (8, 2, 1, 2, 64),
                                                       (80, 40, 33, 40, 16), (9, 3, 3, 1, 16)])
@pytest.mark.parametrize("tokens", [1, 7, 70, 300])
def test_router_over_groups_of_experts(dtype, experts, count, keep, top, ff, tokens):
    """The choice (groups by their two best, then experts), corrections that make choice scores negative, the weights
    without the correction, and the whole feed-forward: both tile sizes and the library's grouped product."""
    from llm_infer_engine_b200.kernels import ops
    hidden = 64
    part, w = build("feed_forward", "routed_experts", {
        "hidden": hidden, "n_experts": experts, "top": top, "expert_ff": ff, "activation": "silu", "router_bias": False,
        "scoring": "sigmoid_groups", "groups": count, "groups_keep": keep}, dtype, seed=experts + top, std=0.3)
    g = torch.Generator().manual_seed(tokens + experts)
    w["correction"] = (torch.randn(experts, generator=g) * 0.5 - 0.6).to(torch.bfloat16).float()
    part.load({k: v.to(DEV, DTYPES[dtype]) for k, v in w.items()})
    x = torch.randn(tokens, hidden, generator=g).to(DTYPES[dtype])
    f = {"router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}
    wd = {k: v.double() for k, v in w.items()}
    chosen, weights = plain.route(x.double(), wd, "", f["router"])
    clear = plain.choice_margin(x.double(), wd, "", f["router"]) > 1e-4
    assert int(clear.sum()) >= tokens * 0.9
    ids = torch.empty(tokens, top, dtype=torch.int32, device=DEV)
    got_w = torch.empty(tokens, top, device=DEV)
    ops.moe_route(x.to(DEV), part.w_router, None, ids, got_w, ops.ROUTE_SIGMOID_GROUPS, part.correction, 1.0, (count, keep))
    order, order_p = ids.cpu().long().sort(dim=1), chosen.sort(dim=1)
    assert torch.equal(order.values[clear], order_p.values[clear])
    assert float((got_w.cpu().double().gather(1, order.indices) - weights.gather(1, order_p.indices))[clear].abs().max()) < 1e-5
    y = part.forward(x.to(DEV), make_ctx([tokens], [0], [0], dtype)).float().cpu().double()
    want = plain.moe(x.double(), wd, "", f)
    assert float((y - want)[clear].abs().max()) <= tol(dtype, float(want.abs().max())) * 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode,rank,n", [("power", 16, 300), ("power", 7, 37), ("double_exp", 11, 128), ("double_exp", 300, 40)])
def test_decays_from_a_low_rank_product(dtype, mode, rank, n):
    """A column slice as input; decays next to 0 and next to 1."""
    from llm_infer_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(rank)
    wide = torch.randn(35, rank + 21, generator=g).to(DTYPES[dtype])
    x = wide[:, 13:13 + rank].double()
    B, bias = torch.randn(n, rank, generator=g) * 2 / rank ** 0.5, torch.linspace(-9, 6 if mode == "power" else 2, n)
    z = (torch.tanh(x) if mode == "double_exp" else x) @ B.T.double() + bias.double()
    want = torch.exp(-torch.exp(z)) if mode == "double_exp" else torch.sigmoid(z) ** (1 / 5.0)
    out = torch.empty(35, n, device=DEV)
    ops.low_rank_gate(wide.to(DEV)[:, 13:13 + rank], B.t().contiguous().to(DEV), bias.to(DEV), out,
                      ops.GATE_DOUBLE_EXP if mode == "double_exp" else ops.GATE_POWER, 5.0)
    assert float((out.cpu().double() - want).abs().max()) < 3e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", [64, 50])
def test_previous_tokens_input_in_pieces(dtype, d):
    """Five mixes of every token with the one before it, across the borders of pieces, in one-token steps too."""
    from llm_infer_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    xs = [torch.randn(n, d, generator=g).to(DTYPES[dtype]) for n in (41, 12)]
    mu = torch.rand(5, d, generator=g)
    want = [torch.stack([plain.shifted_mix(x.double(), m.double()) for m in mu]) for x in xs]
    prev = torch.zeros(4, 1, d, device=DEV)
    prev[2] = 7.0
    held = [0, 0]
    for pieces in ([20, 1], [1, 1], [2, 3], [1, 1], [17, 6]):
        ctx = make_ctx(pieces, held, [3, 1], dtype)
        x = torch.cat([xs[i][held[i]:held[i] + pieces[i]] for i in range(2)]).to(DEV)
        out = torch.empty(5, sum(pieces), d, dtype=DTYPES[dtype], device=DEV)
        ops.shift_mix(x, prev, mu.to(DEV), ctx.cu_q, ctx.tok_seq, ctx.seq_slot, out, single=ctx.decode)
        if not ctx.decode:
            ops.conv_state_store(x, 0, None, prev, ctx.cu_q, ctx.seq_slot, 2)
        ref = torch.cat([want[i][:, held[i]:held[i] + pieces[i]] for i in range(2)], dim=1)
        assert float((out.float().cpu().double() - ref).abs().max()) <= tol(dtype, 4.0), pieces
        held = [h + p for h, p in zip(held, pieces)]
    assert float((prev[2] - 7.0).abs().max()) == 0.0 and float(prev[0].abs().max()) == 0.0


FORMS = ["key_decay", "bonus", "delta"]


def _recurrence_inputs(form, lens, heads, groups, dim, vdim, seed, dtype):
    """Per sequence q, k, v, decays and rates, rounded to the engine's type where the engine hands them over in it; some
    channels remember for hundreds of tokens and some forget at once. And the readings of the plain recurrence."""
    g = torch.Generator().manual_seed(seed)
    dt = DTYPES[dtype]
    seqs = []
    bonus = torch.rand(groups, dim, generator=g)
    for n in lens:
        q, k = torch.randn(n, groups, dim, generator=g), torch.randn(n, groups, dim, generator=g)
        v = torch.randn(n, heads, vdim, generator=g).to(dt).float()
        s = {"v": v}
        if form == "delta":
            s["q"], s["k"] = plain.unit_vector(q) * dim ** -0.5, plain.unit_vector(k + 0.5)
            s["beta"] = torch.rand(n, heads, generator=g)
            s["g"] = 1 - torch.rand(n, heads, generator=g) ** 2 * 0.1
            s["g"][::17] = 1e-3
        else:
            s["q"], s["k"] = q.to(dt).float(), k.to(dt).float()
            a = torch.rand(n, groups, dim, generator=g)
            a[:, :, 0::5] = 1 - a[:, :, 0::5] ** 4 * 0.01
            a[:, :, 1::7] = a[:, :, 1::7] ** 4 * 0.01
            s["a"] = a
        S = torch.zeros(heads, dim, vdim, dtype=torch.float64)
        rows = []
        spread = lambda t: t.double().repeat_interleave(heads // groups, dim=0)              # noqa: E731
        for t in range(n):
            qt, kt, vt = spread(s["q"][t]), spread(s["k"][t]), v[t].double()
            if form == "delta":
                S = s["g"][t].double()[:, None, None] * S
                held = torch.einsum("hdv,hd->hv", S, kt)
                S = S + kt[:, :, None] * (s["beta"][t].double()[:, None] * (vt - held))[:, None, :]
                rows.append(torch.einsum("hdv,hd->hv", S, qt))
                continue
            kv = kt[:, :, None] * vt[:, None, :]
            old = S
            S = spread(s["a"][t])[:, :, None] * S + kv
            rows.append(torch.einsum("hdv,hd->hv", S if form == "key_decay" else old + spread(bonus)[:, :, None] * kv, qt))
        s["want"] = torch.stack(rows).reshape(n, -1)
        seqs.append(s)
    return seqs, bonus


def _scan(form, seqs, bonus, held, pieces, state, slots, heads, groups, dim, vdim, dtype, max_len):
    from llm_infer_engine_b200.kernels import ops
    dt, T = DTYPES[dtype], sum(pieces)
    cat = lambda key: torch.cat([s[key][h:h + p].reshape(p, -1) for s, h, p in zip(seqs, held, pieces)])   # noqa: E731
    cu = [0]
    for p in pieces:
        cu.append(cu[-1] + p)
    cu = torch.tensor(cu, dtype=torch.int32, device=DEV)
    out = torch.empty(T, heads * vdim, device=DEV)
    args = (state, cu, slots, out, len(pieces), heads, groups, dim, vdim)
    if form == "delta":
        q, k = cat("q"), cat("k")
        qk = (q * k).view(T, groups, dim).sum(-1).contiguous().to(DEV)
        scal = torch.stack([cat("beta"), cat("g")], dim=-1).contiguous().to(DEV)
        ops.channel_scan(ops.FORM_DELTA, q.to(DEV), k.to(DEV), cat("v").to(DEV, dt), *args, scal=scal, qk=qk)
    else:
        # q, k and v as columns of one wider tensor, as the projections leave them
        wide = torch.cat([cat("q") * 2, cat("k"), cat("v")], dim=1).to(DEV, dt)
        n = groups * dim
        ops.channel_scan(ops.FORM_KEY_DECAY if form == "key_decay" else ops.FORM_BONUS, wide[:, :n], wide[:, n:2 * n],
                         wide[:, 2 * n:], *args, q_scale=0.5, gate=cat("a").to(DEV),
                         bonus=bonus.reshape(-1).to(DEV) if form == "bonus" else None, max_len=max_len)
    return out.cpu().double()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("heads,groups,dim,vdim", [(3, 3, 20, 24), (6, 2, 9, 10), (2, 2, 64, 64), (4, 2, 36, 44), (2, 1, 128, 33),
                                                   (1, 1, 130, 20), (1, 1, 300, 16), (64, 64, 64, 64)])
def test_recurrences_in_pieces_equal_the_plain_loop(dtype, form, heads, groups, dim, vdim):
    """Three sequences in unequal pieces: single tokens, pieces that end inside, at and behind a tile's edge, and pieces
    long enough for chunks side by side (one a single chunk, one that ends at a chunk's end); another slot's state stays."""
    if form != "delta" and groups != heads:
        groups = heads
    long = heads * dim * vdim < 40000
    plan = [[20, 1, 8], [1, 1, 1], [16, 7, 9]] + ([[260, 128, 129], [1, 1, 1], [300, 256, 5]] if long else [[3, 24, 1]])
    lens = [sum(p[i] for p in plan) for i in range(3)]
    seqs, bonus = _recurrence_inputs(form, lens, heads, groups, dim, vdim, dim + vdim, dtype)
    state = torch.zeros(5, heads, dim, vdim, device=DEV)
    state[2] = 7.0
    slots = torch.tensor([3, 1, 4], dtype=torch.int32, device=DEV)
    held = [0, 0, 0]
    for pieces in plan:
        got = _scan(form, seqs, bonus, held, pieces, state, slots, heads, groups, dim, vdim, dtype, max(pieces))
        ref = torch.cat([s["want"][h:h + p] for s, h, p in zip(seqs, held, pieces)])
        assert float((got - ref).abs().max()) <= 2e-5 * max(1.0, float(ref.abs().max())), pieces
        held = [h + p for h, p in zip(held, pieces)]
    assert float((state[2] - 7.0).abs().max()) == 0.0 and float(state[0].abs().max()) == 0.0


@pytest.mark.parametrize("form", FORMS)
def test_a_long_pieces_chunks_give_what_the_whole_piece_gives(form):
    """The same long piece whole, in chunks, and beside other sequences; float32 rows beside other sequences are the same
    bits."""
    heads, dim, vdim = 2, 40, 24
    seqs, bonus = _recurrence_inputs(form, [700, 300], heads, heads, dim, vdim, 5, "float32")
    outs = []
    for n, max_len in ((1, None), (1, 700), (2, 700)):
        state = torch.zeros(4, heads, dim, vdim, device=DEV)
        slots = torch.tensor([2, 1][:n], dtype=torch.int32, device=DEV)
        got = _scan(form, seqs[:n], bonus, [0] * n, [700, 300][:n], state, slots, heads, heads, dim, vdim, "float32", max_len)
        outs.append((got[:700], state[2].clone()))
    assert float((outs[0][0] - outs[1][0]).abs().max()) <= 1e-5 * float(outs[0][0].abs().max())
    assert torch.equal(outs[1][0], outs[2][0]) and torch.equal(outs[1][1], outs[2][1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,groups,dim,vdim", [(3, 3, 20, 24), (6, 2, 9, 10), (4, 2, 64, 64), (2, 1, 128, 128), (1, 1, 300, 16)])
def test_unit_vectors_rates_and_decays_of_the_delta_rule(dtype, heads, groups, dim, vdim):
    from llm_infer_engine_b200.kernels import ops
    g = torch.Generator().manual_seed(dim)
    T = 21
    qkv = torch.randn(T, 2 * groups * dim + heads * vdim, generator=g).to(DTYPES[dtype])
    qkv[3, :dim] = 1e-4                                               # next to the constant under the root
    ba = torch.randn(T, 2 * heads + 5, generator=g).to(DTYPES[dtype])
    A, dt = torch.rand(heads, generator=g) * 4, torch.randn(heads, generator=g)
    f32 = dict(dtype=torch.float32, device=DEV)
    qn, kn = torch.empty(T, groups * dim, **f32), torch.empty(T, groups * dim, **f32)
    scal, qk = torch.empty(T, heads, 2, **f32), torch.empty(T, groups, **f32)
    ops.delta_prepare(qkv.to(DEV), ba.to(DEV), 5, 5 + heads, A.to(DEV), dt.to(DEV), 1e-6, 0.3, qn, kn, scal, qk, heads, groups, dim)
    x = qkv.double()
    q, k = x[:, :groups * dim].view(T, groups, dim), x[:, groups * dim:2 * groups * dim].view(T, groups, dim)
    q, k = plain.unit_vector(q) * 0.3, plain.unit_vector(k)
    assert float((qn.cpu().double() - q.reshape(T, -1)).abs().max()) < 1e-6
    assert float((kn.cpu().double() - k.reshape(T, -1)).abs().max()) < 1e-6
    assert float((qk.cpu().double() - (q * k).sum(-1)).abs().max()) < 1e-6
    b, a = ba.double()[:, 5:5 + heads], ba.double()[:, 5 + heads:5 + 2 * heads]
    assert float((scal[:, :, 0].cpu().double() - torch.sigmoid(b)).abs().max()) < 1e-6
    assert float((scal[:, :, 1].cpu().double() - torch.exp(-A.double() * plain.softplus(a + dt.double()))).abs().max()) < 1e-6


# ------------------------------------------------------------------------------------------ parts alone
def _run_mixer_in_pieces(mixer, cache, dtype, xs, want, schedule):
    slots = [cache.take_slot() for _ in xs]
    held = [0] * len(xs)
    for pieces in schedule:
        live = [i for i, p in enumerate(pieces) if p > 0]
        for i in live:
            cache.reserve(slots[i], held[i] + pieces[i])
        ctx = make_ctx([pieces[i] for i in live], [held[i] for i in live], [slots[i] for i in live], dtype,
                       kernels=kernel_plan(dtype))
        x = torch.cat([xs[i][held[i]:held[i] + pieces[i]] for i in live])
        y = mixer.forward(x.to(DEV), ctx, cache.unit(0), True)
        if hasattr(y, "terms"):
            ts = [t.float().cpu().double() for t, _ in y.terms]
            if y.term_norms:
                ts = [plain.rms_unit(t, y.term_norms[1]) * v.cpu().double() for t, v in zip(ts, y.term_norms[0])]
            y = sum(c * t for t, (_, c) in zip(ts, y.terms))
        y = y.float().cpu().double()
        ref = torch.cat([want[i][held[i]:held[i] + pieces[i]] for i in live])
        # a reading next to zero (a query across its key) is divided by its own size: bfloat16 inputs then show more
        slack = 2 if dtype == "float32" else 5
        assert float((y - ref).abs().max()) <= tol(dtype, float(ref.abs().max())) * slack, (pieces, held)
        for i in live:
            held[i] += pieces[i]
            cache.note_appended(slots[i], held[i], device_updated=False)
    return slots


def _mixer_weights(w, seed):
    """Vectors and decays as a design would have them: long memories, taps of both signs, a bonus that counts."""
    g = torch.Generator().manual_seed(seed)
    for name in w:
        last = name.split(".")[-1]
        shape = w[name].shape
        if last == "conv":
            w[name] = torch.randn(shape, generator=g) * 0.6
        elif last == "dt_bias":
            w[name] = torch.rand(shape, generator=g) * 3 - 5
        elif last == "A_log":
            w[name] = torch.rand(shape, generator=g) * 1.5 - 1
        elif last == "w0":
            w[name] = torch.rand(shape, generator=g) * 6 - 6
        elif name.endswith("a2.b"):
            w[name] = torch.rand(shape, generator=g) * 4 - 1
        w[name] = w[name].to(torch.bfloat16).float()
    return w


def _spec(tag, layer):
    from llm_infer_engine_b200.config import load_config
    arch, cfg = load_config(CFGS[tag])
    return arch.to_spec(cfg).layers[layer].mixer


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag,layer", [("a", 0), ("a", 1), ("a", 2), ("a", 3), ("b", 0), ("b", 1), ("b", 2), ("c", 0), ("c", 1),
                                       ("c", 2)])
def test_mixers_in_pieces(dtype, tag, layer):
    """Every kind of mixer as a part: two sequences over prompts in pieces (shorter than the convolution's reach, and long
    enough for chunks), single tokens, and a slot that is given back and taken again, whose states must start at zero."""
    from llm_infer_engine_b200.cache import Cache
    cfg = CFGS[tag]
    spec, entry = _spec(tag, layer), cfg["layers"][layer]
    mixer, w = build("mixer", spec.kind, spec.params, dtype, seed=layer + 5, std=0.2)
    w = _mixer_weights(w, layer)
    mixer.load({k: v.to(DEV, DTYPES[dtype]) for k, v in w.items()})
    wd = {k: v.double() for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    plain_mixer = lambda x: plain.MIXERS[entry["type"]](x.double(), wd, "", entry["mixer"], eps)       # noqa: E731
    cache = Cache([mixer.cache_requests()], 3, 64 * 24, 1024, DTYPES[dtype], DEV)
    cache.take_slot()
    g = torch.Generator().manual_seed(11)
    xs = [torch.randn(n, cfg["width"], generator=g).to(DTYPES[dtype]) for n in (440, 72)]
    slots = _run_mixer_in_pieces(mixer, cache, dtype, xs, [plain_mixer(x) for x in xs],
                                 ([1, 2], [2, 1], [100, 30], [295, 2], [1, 1], [1, 1], [40, 35]))
    cache.give_back_slot(slots[1])
    xs2 = [torch.randn(70, cfg["width"], generator=g).to(DTYPES[dtype])]
    _run_mixer_in_pieces(mixer, cache, dtype, xs2, [plain_mixer(xs2[0])], ([2], [67], [1]))


# ------------------------------------------------------------------------------------------ the attention's edges
def _edge_case(dtype, hd, hdv, n_q, n_kv, window, n, q_len, probe):
    """A sequence of n keys of which the last q_len are this step's queries; the LAST query points straight at key
    `probe`, whose value is a marker (50 in every entry), so that its softmax weight is next to one when it is visible.
    Slots and pages were given back and taken again before, so the sequence's pages are out of order."""
    from llm_infer_engine_b200.cache import Cache, KVRequest
    from llm_infer_engine_b200.parts import AttentionOptions
    cache = Cache([[KVRequest(n_kv, hd, window, v_head_dim=hdv)]], 4, 64 * 24, 1024, DTYPES[dtype], DEV)
    cache.take_slot()
    other = cache.take_slot()
    cache.reserve(other, 130)
    slot = cache.take_slot()
    cache.reserve(slot, 70)
    cache.give_back_slot(other)
    cache.reserve(slot, n)
    g = torch.Generator().manual_seed(n * 7 + probe)
    k = torch.randn(n, n_kv, hd, generator=g) * 0.3
    v = torch.randn(n, n_kv, hdv, generator=g) * 0.1
    q = torch.randn(q_len, n_q, hd, generator=g) * 0.3
    direction = torch.nn.functional.normalize(torch.randn(hd, generator=g), dim=0)
    k[probe] += direction * 8.0
    q[-1] = direction * 8.0
    v[probe] = 50.0
    k, v, q = (t.to(DTYPES[dtype]) for t in (k, v, q))
    kv = cache.unit(0).kv
    table = kv.block_table[slot].cpu()
    for j in range(n):
        kv.k[int(table[j // 64]), :, j % 64] = k[j].to(DEV)
        kv.v[int(table[j // 64]), :, j % 64] = v[j].to(DEV)
    ctx = make_ctx([q_len], [n - q_len], [slot], dtype, kernels=kernel_plan(dtype))
    out = torch.empty(q_len, n_q * hdv, dtype=DTYPES[dtype], device=DEV)
    ctx.attention(q.reshape(q_len, -1).to(DEV), kv, out, n_q, n_kv, hd, AttentionOptions(scale=0.5, window=window))
    ok = plain.window_visible(n, window)[n - 1]
    want = []
    for h in range(n_q):
        kh = k[:, h // (n_q // n_kv)].double()
        a = torch.softmax((q[-1, h].double() @ kh.T * 0.5).masked_fill(~ok, float("-inf")), dim=-1)
        want.append(a @ v[:, h // (n_q // n_kv)].double())
    return out[-1].float().cpu(), torch.cat(want).float(), bool(ok[probe])


EDGES = [  # window, keys, probe, may the last query (position keys - 1) see it
    (80, 300, 220, True), (80, 300, 219, False),          # just inside and just outside the window
    (64, 257, 193, True), (64, 257, 192, False),          # the window's edge on a page's edge
    (65, 257, 192, True), (65, 257, 191, False),
    (0, 500, 3, True), (0, 700, 0, True),                 # no window: keys far back, the first token
    (1, 40, 39, True), (1, 40, 38, False), (2, 130, 128, True), (2, 130, 127, False),
    (300, 90, 0, True), (128, 129, 1, True), (128, 129, 0, False)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(24, 40, 4, 2), (64, 64, 6, 1), (128, 128, 2, 2), (32, 16, 6, 3), (48, 112, 4, 2)])
@pytest.mark.parametrize("q_len", [1, 2, 37, 200])
def test_keys_at_every_edge_of_a_window_stand_out(dtype, shape, q_len):
    """A probe key that the query may see puts the marker into the output (about 50); one that it may not see leaves
    the output small. Every attention kernel, value heads narrower and wider than key heads included."""
    hd, hdv, n_q, n_kv = shape
    for window, n, probe, visible in EDGES:
        if q_len > n:
            continue
        got, want, ok = _edge_case(dtype, hd, hdv, n_q, n_kv, window, n, q_len, probe)
        assert ok == visible
        assert float((got - want).abs().max()) <= (1e-3 if dtype == "float32" else 0.6), (window, n, probe)
        assert (float(got.abs().max()) > 25) == visible, (window, n, probe, float(got.abs().max()))


# ------------------------------------------------------------------------------------------ the engine
@pytest.mark.parametrize("tag,dtype", [(t, d) for t in ("a", "b", "c") for d in ("float32", "bfloat16")] + [("routed", "float32")])
def test_every_schedule_matches_plain(tag, dtype):
    """Whole prompts; the last tokens one by one (more of them than the longest window); unequal batches in which
    shorter requests end early and the next batch takes their slots, pages and states; prompts in pieces of 2, 7, 64
    and 100 tokens; a prompt in pieces beside sequences that go on by one token."""
    requests = requests_for(tag)
    want = oracle(tag, requests)
    engine = engine_for(tag, dtype)
    plans = {"whole": helpers.plan_whole(requests), "tail": helpers.plan_tail(requests, 120),
             "batched": helpers.plan_batched(requests, 3, 0.6), "mixed": helpers.plan_mixed(requests, 9)}
    some = {rid: toks for rid, toks in requests.items() if len(toks) <= 200}
    for chunk in (2, 7, 64, 100):
        plans[f"pieces of {chunk}"] = helpers.plan_chunked(some if chunk == 2 else requests, chunk)
    for name, steps in plans.items():
        got = helpers.run_plan_engine(engine, steps)
        compare(got, {rid: want[rid] for rid in got}, dtype, f"{tag}/{dtype}/{name}", tag)
        assert engine.cache.free_slots() == engine.cache.n_slots and engine.cache.free_pages() == engine.cache.n_pages
    if dtype == "bfloat16":
        from llm_infer_engine_b200.kernels import ops
        ops.check_tc_status("cuda")


@pytest.mark.parametrize("tag", ["a", "b", "c"])
def test_the_models_are_sharp_enough_to_show_what_a_fault_would_change(tag):
    """The bounds above mean something only if a fault moves the logits by more than they allow. In the plain
    implementation each of these differs by more than a bfloat16 bound at more positions than are forgiven."""
    w, cfg = plain_weights(tag), CFGS[tag]
    toks = helpers.random_tokens(cfg["vocab"], max(LENGTHS[tag]), seed=47)
    right = plain.forward(w, cfg, toks)
    tol_ = bound("bfloat16", right)

    def gap(what, cfg2=cfg, w2=w):
        diff = (plain.forward(w2, cfg2, toks) - right).abs().max(dim=1).values
        assert int((diff > tol_).sum()) > max(1, len(diff) // 25) and float(diff.max()) > 1.5 * tol_, (
            tag, what, int((diff > tol_).sum()), float(diff.max()), tol_)

    def changed(suffix, f):
        return {k: (f(v) if k.endswith(suffix) else v) for k, v in w.items()}

    def edited(f):
        c = json.loads(json.dumps(cfg))
        for layer in c["layers"]:
            f(layer, layer["mixer"], layer["mlp"])
        return c

    def window(layer, m, f):
        if layer["type"] != "delta" and m["left"]["mask"]:
            m["left"]["mask"]["size"] += 1

    def rotation(layer, m, f):
        if layer["type"] == "parallel_2":
            m["left"]["rot"]["base"] *= 3

    def root(layer, m, f):
        if layer["type"] == "parallel":
            m["right"]["tau"] *= 3

    def limit(layer, m, f):
        if f and f["kind"] == "dense":
            f["limit"] *= 4

    def groups(layer, m, f):
        if f and f["kind"] == "moe":
            f["router"]["groups"]["keep"] = f["router"]["groups"]["count"]

    gap("window", edited(window))
    gap("rotation", edited(rotation))
    gap("root of the decay", edited(root))
    gap("limit", edited(limit))
    if tag != "b":                                                    # its one group is always kept, all experts used
        gap("groups", edited(groups))
        gap("correction", w2=changed(".correction", torch.zeros_like))
    if cfg["loop"]:
        gap("loop", dict(cfg, loop=dict(cfg["loop"], times=cfg["loop"]["times"] - 1)))
    gap("branch constant", dict(cfg, residual_mult=cfg["residual_mult"] * 1.2))
    gap("gate per head", w2=changed(".left.g", torch.zeros_like))
    gap("bonus", w2=changed(".right.u", torch.zeros_like))
    gap("previous token", w2={k: (v * 0 if ".mu." in k else v) for k, v in w.items()})
    gap("forgetting at once, key decay", w2=changed(".a2.b", lambda v: v - 9 * 16))
    gap("forgetting at once, time mixing", w2=changed(".w0", lambda v: v + 6))
    gap("forgetting at once, delta rule", w2=changed(".dt_bias", lambda v: v + 9))
    gap("rate", w2=changed(".mix.b", torch.zeros_like))
    gap("order of taps", w2={k: (v.flip(1) if k.endswith(".conv") else v) for k, v in w.items()})
    gap("norm behind a branch", w2=changed(".norm1b", torch.zeros_like))
    gap("norm of a mixer of two", w2=changed(".left.out", torch.ones_like))
    gap("norm of the delta rule", w2=changed(".mix.norm", torch.ones_like))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batch_and_cutting_do_not_change_a_row(dtype):
    """The logits of a position do not depend on what else is in the batch or how the prompt was cut: float32
    kernels sum in a fixed order, so there the rows are equal bit for bit."""
    tag = "a"
    requests = requests_for(tag)
    engine = engine_for(tag, dtype)
    alone = helpers.run_plan_engine(engine, helpers.plan_whole(requests))
    together = helpers.run_plan_engine(engine, helpers.plan_batched(requests, 8, 1.0))
    pieces = helpers.run_plan_engine(engine, helpers.plan_chunked(requests, 7))
    for rid in requests:
        if dtype == "float32":
            # (a prompt of one token alone is a one-token step, which has kernels of its own)
            assert len(requests[rid]) == 1 or torch.equal(alone[rid], together[rid]), rid
            assert float((alone[rid] - together[rid]).abs().max()) <= 0.2 * bound(dtype, alone[rid]), rid
            assert float((alone[rid] - pieces[rid]).abs().max()) <= 0.2 * bound(dtype, alone[rid]), rid
        else:
            assert float((alone[rid] - together[rid]).abs().max()) <= bound(dtype, alone[rid])


def test_a_prompt_length_that_comes_again_is_captured_and_replayed():
    """A lone prompt of a length seen before runs as one graph: slots with states of their own, other tokens."""
    tag = "c"
    engine = engine_for(tag, "bfloat16", max_batch=3, max_tokens=64 * 12, cuda_graph=True)
    for seed in range(4):
        requests = {"x": helpers.random_tokens(CFGS[tag]["vocab"], 129, seed=90 + seed)}
        got = helpers.run_plan_engine(engine, helpers.plan_whole(requests))
        compare(got, oracle(tag, requests), "bfloat16", f"prompt {seed}", tag)


def test_trace_run_program_and_other_sizes_at_once(tmp_path):
    """bin/trace_run as a subprocess on the configuration with the odd sizes."""
    tag = "b"
    requests = {k: v for k, v in requests_for(tag).items() if len(v) <= 200}
    want = oracle(tag, requests)
    steps = helpers.plan_batched(requests, 4, 0.5)
    peak = max(sum(len(v) for v in requests.values()), 64)
    for dtype in ("float32", "bfloat16"):
        got = helpers.run_plan_trace_run(folder_for(tag), dtype, steps, peak, CFGS[tag]["vocab"])
        compare(got, want, dtype, f"trace_run/{dtype}", tag)


@pytest.mark.parametrize("dtype,gap", [("float32", 1e-4), ("bfloat16", 2.0)])
@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation_through_the_library(dtype, gap, graph):
    """generate(): admission, ragged prompts, captured one-token steps (the recurrences, the routed feed-forward's sort
    inside), slots and their states used again. Greedy tokens equal the plain implementation's; where they part the two
    candidates are close in the plain logits (by what the bfloat16 engine may differ from them)."""
    from llm_infer_engine_b200 import GenerationStats, generate
    tag = "a"
    w, cfg = plain_weights(tag), CFGS[tag]
    prompts = [helpers.random_tokens(cfg["vocab"], n, seed=60 + i) for i, n in enumerate([1, 5, 42, 64, 3, 90, 2])]
    engine = engine_for(tag, dtype, max_batch=3, max_tokens=64 * 12, cuda_graph=graph)
    stats = GenerationStats()
    out = generate(engine, prompts, max_new_tokens=40, stop_ids=[], stats=stats)          # decoding crosses the window
    assert stats.batches >= 3 and [len(o) for o in out] == [40] * len(prompts)
    same = total = 0
    for p, o in zip(prompts, out):
        rows = plain.forward(w, cfg, list(p) + list(o[:-1]))[len(p) - 1:]
        for i, (row, tok) in enumerate(zip(rows, o)):
            best = int(row.argmax())
            total, same = total + 1, same + (tok == best)
            if tok != best:
                assert float(row[best] - row[tok]) < gap, (len(p) + i, tok, best)
    assert same >= (total if dtype == "float32" else 0.9 * total)
    engine.cache.check()
    assert engine.cache.free_slots() == 3 and engine.cache.free_pages() == engine.cache.n_pages


def test_long_decoding_in_float32():
    """A few hundred captured one-token steps against one whole-sequence pass: the windows pass over decoded tokens
    many times and the states are carried through every step."""
    from llm_infer_engine_b200 import generate
    tag = "b"
    w, cfg = plain_weights(tag), CFGS[tag]
    prompt = helpers.random_tokens(cfg["vocab"], 4, seed=70)
    engine = engine_for(tag, "float32", max_batch=2, max_tokens=64 * 12, cuda_graph=True)
    out = generate(engine, [prompt, prompt[:1]], max_new_tokens=260, stop_ids=[])
    for p, o in zip([prompt, prompt[:1]], out):
        seq = p + o
        ref = plain.forward(w, cfg, seq[:-1])
        picks = ref[len(p) - 1:].argmax(-1).tolist()
        for i, (a, b) in enumerate(zip(o, picks)):
            if a != b:
                row = ref[len(p) - 1 + i]
                assert float(row[b] - row[a]) < 1e-4, (i, a, b)
                break


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
        row = plain.forward(w, cfg, seq)[-1]
        assert tok == int(row.argmax()) or float(row.max() - row[tok]) < 1e-4
        seq.append(tok)
    assert len(ids) == 6

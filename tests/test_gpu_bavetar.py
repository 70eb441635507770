"""The Bavetar decoder in the engine against the plain implementation (tests/plain_bavetar.py): every mechanism
alone, then whole models under every way of cutting and batching the work, in float32 and bfloat16.  The tiny
models and their weights are made here."""
import numpy as np
import pytest
import torch

import plain_bavetar as plain
from helpers import (max_live_tokens, random_tokens, replay_in_process, schedule_mixed, schedule_portions, schedule_tail,
                     schedule_whole)
from test_gpu_dugudra import edge_case
from test_gpu_linurax import close, ctx_of, fill
from test_gpu_nufatar import filled, run_attention, set_weight
from test_gpu_sapatar import named, row_error, run_state_mixer
from tiny_bavetar import BAVETAR_CONFIGS, BAVETAR_E, BAVETAR_PAGE, BAVETAR_SEEDS, BAVETAR_STD, dense, latent, mamba, moe

import tessweave_engine_b200 as tw
from tessweave_engine_b200.config.bavetar_config import BavetarConfig
from tessweave_engine_b200.csrc import ops
from tessweave_engine_b200.csrc.ops import SplitSum
from tessweave_engine_b200.models.bavetar import feed_forward_spec, mixer_spec
from tessweave_engine_b200.parts import PartSpec, ResidualStream, Runtime, build_part, dense_delta
from tessweave_engine_b200.parts.base import DeltaPair

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def typed_layer(width, layer, eps=1e-5):
    """The typed configuration of a model of one layer, and that layer."""
    typed = BavetarConfig.from_dict({"vocab": 8, "width": width, "norm": {"eps": eps}, "layers": [layer]})
    return typed, typed.layers[0]


def mixer_of(rt, width, layer, eps=1e-5):
    typed, one = typed_layer(width, layer, eps)
    return build_part("mixer", mixer_spec(typed, one), rt)


# ---------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------
def delta_of(kind, rows, hidden, g, dtype):
    """(what the kernel is given, its value in fp32)"""
    if kind == "none":
        return None, torch.zeros(rows, hidden)
    if kind == "dense":
        d = torch.randn(rows, hidden, generator=g).to(dtype)
        return d.cuda(), d.float()
    slices = torch.randn(int(kind), rows, hidden, generator=g)
    return SplitSum(slices.cuda()), slices.sum(0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,rows", [(40, 5), (36, 70), (37, 3), (192, 300), (1024, 8), (2050, 3), (4100, 70), (8500, 2)])
@pytest.mark.parametrize("first,second", [("dense", "dense"), ("3", "dense"), ("dense", "5"), ("18", "2"), ("none", "none"), ("dense", "none"), ("none", "4")])
def test_two_deltas_in_two_norms_out(dtype, hidden, rows, first, second):
    """x <- x + (d1 + d2) in 32 bits and two normalised copies with weights of their own: every form of the kernel (rows
    in registers, read twice, four values per thread, a cluster per row), every kind of delta, chosen rows, one copy."""
    g = torch.Generator().manual_seed(hidden + rows)
    resid = torch.randn(rows, hidden, generator=g)
    d1, v1 = delta_of(first, rows, hidden, g, dtype)
    d2, v2 = delta_of(second, rows, hidden, g, dtype)
    w1, w2 = (1 + 0.3 * torch.randn(hidden, generator=g) for _ in range(2))
    x = resid.double() + (v1.double() + v2.double())
    want1, want2 = ((plain.rms(x, 1e-5) * w.double()).float() for w in (w1, w2))
    r = resid.cuda().clone()
    a, b = (torch.empty(rows, hidden, dtype=dtype, device="cuda") for _ in range(2))
    ops.add_rmsnorm_pair(a, b, r, d1, d2, w1.cuda(), w2.cuda(), 1e-5, rows)
    assert float((r.cpu().double() - x).abs().max()) <= 2e-6 * float(x.abs().max())
    close(a.float().cpu(), want1, dtype, "first copy", bf16=1e-2)
    close(b.float().cpu(), want2, dtype, "second copy", bf16=1e-2)
    picked = torch.tensor([rows - 1, 0], dtype=torch.int32)
    r = resid.cuda().clone()
    c = torch.empty(2, hidden, dtype=dtype, device="cuda")
    ops.add_rmsnorm_pair(c, None, r, d1, d2, w2.cuda(), None, 1e-5, 2, rows=picked.cuda())
    assert torch.equal(r.cpu(), resid)                  # with chosen rows the stream is left as it was
    close(c.float().cpu(), want2[picked.long()], dtype, "chosen rows", bf16=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_block_with_two_norms(dtype):
    """x + (mixer(norm1 x) + feed_forward(norm2 x)), both of the same x; norms that differ by more than any rounding."""
    width, rt = 48, Runtime(torch.device("cuda"), dtype)
    layer = mamba(2, 12, 16, 1, 3, 2, dense(40))
    typed, one = typed_layer(width, layer)
    norm = PartSpec("rmsnorm", {"size": width, "eps": 1e-5, "weight_name": ""})
    block = build_part("block", PartSpec("parallel_pre_norm", {
        "hidden": width, "norm1": norm, "norm2": norm, "mixer": mixer_spec(typed, one), "feed_forward": feed_forward_spec(typed, one.mlp),
        "names": {"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feed_forward": "mlp"}}), rt)
    w = fill(block, 5, 0.3)
    for name, seed in (("norm1", 1), ("norm2", 2)):
        w[name] = torch.randn(width, generator=torch.Generator().manual_seed(seed)).to(torch.bfloat16).float()
        getattr(block, name).weight.copy_(w[name])
    wd = {k: v.double() for k, v in w.items()}
    x = torch.randn(9, width, generator=torch.Generator().manual_seed(3))
    ctx = ctx_of(rt, list(range(9)), [0] * 9, [0], [0], [9], [9])
    from tessweave_engine_b200.parts import StateView
    stream = ResidualStream(resid=x.cuda().clone())
    block.forward(ctx, stream, StateView(torch.zeros(1, block.cache_need().numel, device="cuda")), True)
    assert isinstance(stream.pending, DeltaPair)
    got = x + sum(dense_delta(ctx, d, dtype, "t").float().cpu()[:9] for d in (stream.pending.first, stream.pending.second))
    xd = x.double()
    want = xd + (plain.mixer_mamba2(plain.rms(xd, 1e-5) * wd["norm1"], wd, "mix.", layer["mixer"], 1e-5)
                 + plain.dense(plain.rms(xd, 1e-5) * wd["norm2"], wd, "mlp."))
    close(got, want.float(), dtype, "block")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scale,cap", [(2.0, 2.5), (0.3, None), (1.0, 1.5), (-1.5, 4.0)])
def test_scaled_and_capped_logits(dtype, scale, cap):
    rt = Runtime(torch.device("cuda"), dtype)
    head = build_part("head", PartSpec("linear_head", {"vocab": 77, "hidden": 48, "weight_name": "", "softcap": cap, "scale": scale}), rt)
    w = fill(head, 3, 0.6)
    y = torch.randn(9, 48, generator=torch.Generator().manual_seed(1)).to(dtype)
    ctx = ctx_of(rt, list(range(9)), [0] * 9, [0], [0], [9], [9])
    logits = torch.empty(9, 77, dtype=torch.float32, device="cuda")
    head.forward(ctx, logits, y.cuda(), 9)
    want = (y.double() @ w[""].double().T) * scale
    if cap is not None:
        assert float(want.abs().max()) > cap            # the cap is felt
        want = cap * torch.tanh(want / cap)
    close(logits.cpu(), want.float(), dtype, "logits")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,parts,rows", [(48, 1, 5), (48, 4, 3), (45, 3, 7), (64, 64, 2), (512, 2, 70), (2048, 1, 4), (4096, 2, 3), (7168, 1, 5), (9000, 1, 2)])
def test_gate_before_the_norm_of_parts(dtype, width, parts, rows):
    """u = y silu(z), then every part of u over its own root mean square: parts of one value, parts in registers, parts too
    wide for them; the gate is a column slice of wider rows."""
    g = torch.Generator().manual_seed(width)
    raw = torch.randn(rows, width, generator=g) * torch.rand(1, width, generator=g) * 4
    z = torch.randn(rows, width + 8, generator=g).to(dtype)
    weight = 1 + 0.3 * torch.randn(width, generator=g)
    out = torch.empty(rows, width, dtype=dtype, device="cuda")
    ops.gate_part_norm(out, raw.cuda(), weight.cuda(), z.cuda()[:, 8:], ops.GATE_SILU, 1e-3, rows, parts)
    u = raw.double() * plain.silu(z.double()[:, 8:])
    want = (plain.rms(u.view(rows, parts, -1), 1e-3).reshape(rows, width) * weight.double()).float()
    close(out.float().cpu(), want, dtype, "gated norm", bf16=1e-2)


LATENT_SHAPES = [  # hidden, heads, plain size, rotated size, value size, q latent, kv latent, page, base
    (48, 3, 16, 8, 24, 20, 40, 8, 1000.0), (40, 5, 6, 2, 7, 5, 11, 4, 10.0), (64, 4, 32, 16, 32, 64, 48, 16, 3e4),
    (32, 1, 8, 4, 8, 8, 12, 4, 50.0), (96, 12, 16, 16, 8, 32, 112, 16, 3e5), (64, 9, 24, 32, 16, 48, 96, 16, 1e4),
    (64, 2, 8, 8, 8, 24, 24, 8, 5e4), (64, 2, 16, 8, 16, 24, 300, 16, 1e4), (64, 6, 16, 64, 16, 24, 192, 64, 1e5)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_latent_attention_with_sinks_and_gates_alone(dtype, shape):
    """Queries and keys/values through their latents, the shared rotated key part, a sink per head that takes much of the
    weight, a gate per head; two requests side by side in portions and single tokens."""
    hidden, heads, d, r, dv, qr, cr, page, base = shape
    rt = Runtime(torch.device("cuda"), dtype)
    layer = latent(heads, d, r, dv, qr, cr, 1.5 / (d + r) ** 0.5, base)
    mixer = mixer_of(rt, hidden, layer)
    need = mixer.cache_need()
    assert (need.kv_heads, need.head_dim, need.values_are_keys, need.window) == (1, cr + r, True, None)
    w = filled(mixer, 16, 1.2 / hidden ** 0.5)
    g = torch.Generator().manual_seed(8)
    for name, fan_in in (("uq", qr), ("uk", cr), ("uv", cr)):          # the maps out of the latents keep what passes at size 1
        set_weight(mixer, w, name, torch.randn(w[name].shape, generator=torch.Generator().manual_seed(fan_in)) / fan_in ** 0.5)
    set_weight(mixer, w, "sink", 2.0 + 2.0 * torch.randn(heads, generator=g))
    set_weight(mixer, w, "g", 3.0 * torch.randn(heads, hidden, generator=g) / hidden ** 0.5)
    wd = {k: v.double() for k, v in named(w).items()}
    rows_of = {"a": torch.randn(190, hidden, generator=g).to(dtype), "b": torch.randn(60, hidden, generator=g).to(dtype)}
    plan = [{"a": na, "b": nb} for na, nb in [(0, 19), (13, 1), (150, 0), (1, 1), (1, 38), (2, 1), (1, 0), (22, 0)]]
    got = run_attention(rt, mixer, page, rows_of, plan, poison=True)
    for name, rows in rows_of.items():
        run = lambda weights: plain.mixer_latent_attention(rows.double(), weights, "p.", layer["mixer"], 1e-5, torch.arange(len(rows))).float()   # noqa: E731
        want = run(wd)
        close(got[name], want, dtype, f"request {name}")
        for wrong in ({"p.sink": torch.full_like(wd["p.sink"], -40.0)}, {"p.g": -wd["p.g"]}, {"p.sink": wd["p.sink"] * layer["mixer"]["scale"]}):
            assert float((run({**wd, **wrong}) - want).abs().max()) > 0.1 * float(want.abs().max())     # each term shows


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page,cr,r", [(8, 24, 8), (16, 48, 16), (4, 20, 4)])
def test_one_far_key_of_hundreds(dtype, page, cr, r):
    """One key answers the last token's query far above all others and carries a value of its own: at the first tokens, on
    both sides of page borders, in the middle, next to the end; the asking token comes in a portion and alone.  A key
    that is missed, or a sink that is left out (it has a quarter of the weight), moves the output by its size."""
    rt = Runtime(torch.device("cuda"), dtype)
    hidden, heads, d, dv, qr = 48, 2, 16, 24, 12
    g = torch.Generator().manual_seed(1)
    layer = latent(heads, d, r, dv, qr, cr, 9.0 / d, 1000.0)
    mixer = mixer_of(rt, hidden, layer)
    w = filled(mixer, 8, 0.02)
    # the query latent reads channel 2, the first half of the key/value latent channel 0 (+-1 in every value after their
    # norms), the second half channel 1 (the payload, +-1 too); the maps out of the latents average, the rotated parts are silent
    t = torch.zeros_like(w["dq"]); t[:, 2] = 1.0
    set_weight(mixer, w, "dq", t)
    t = torch.zeros_like(w["dkv"]); t[:cr // 2, 0] = 1.0; t[cr // 2:cr, 1] = 1.0
    set_weight(mixer, w, "dkv", t)
    t = torch.zeros(heads, d + r, qr); t[:, :d, :] = 1.0 / qr
    set_weight(mixer, w, "uq", t.reshape(heads * (d + r), qr))
    t = torch.zeros_like(w["uk"]); t[:, :cr // 2] = 2.0 / cr
    set_weight(mixer, w, "uk", t)
    t = torch.randn(w["uv"].shape, generator=g) * 0.5; t[:, :cr // 2] = 0.0
    set_weight(mixer, w, "uv", t)
    set_weight(mixer, w, "g", torch.zeros_like(w["g"]))
    set_weight(mixer, w, "sink", torch.full((heads,), 8.0))          # the marked key scores 9, the sink 8
    set_weight(mixer, w, "dq.norm", torch.ones(qr)); set_weight(mixer, w, "dkv.norm", torch.ones(cr))
    set_weight(mixer, w, "o", torch.randn(w["o"].shape, generator=g) * 0.3)
    wd = {k: v.double() for k, v in named(w).items()}
    length = 301
    last = length - 1
    base = 0.01 * torch.randn(length, hidden, generator=g)
    base[:, 0], base[:, 1], base[:, 2] = -1.0, 1.0, 1.0
    run = lambda h, weights=wd: plain.mixer_latent_attention(h.double(), weights, "p.", layer["mixer"], 1e-5, torch.arange(length)).float()[-1:]   # noqa: E731
    quiet = run(base.to(dtype))
    for j in (0, 1, page - 1, page, 4 * page - 1, 4 * page, 127, 128, 150, last - page, last - 1):
        h = base.clone()
        h[j, 0], h[j, 1] = 1.0, -1.0
        h = h.to(dtype)
        want = run(h)
        size = float(torch.maximum(want.abs().max(), quiet.abs().max()))
        assert float((want - quiet).abs().max()) > 0.3 * size            # the marked key shows
        assert float((run(h, {**wd, "p.sink": torch.full((heads,), -50.0, dtype=torch.float64)}) - want).abs().max()) > 0.1 * size
        for tail in (0, 1, 9):                                           # the asking token inside a portion, alone, after single tokens
            err = float((edge_case(rt, mixer, page, h, tail) - want).abs().max())
            assert err <= (2e-5 if dtype == torch.float32 else 0.1) * size, f"key at {j}, last {tail} tokens alone: {err:.3g} of {size:.3g}"


LATENT_TC5 = [  # row, value columns, heads, page, window, portions as (rows of this step, rows held before)
    (256, 192, 28, 16, None, [(300, 0), (97, 411), (1, 50)]), (128, 96, 6, 16, None, [(129, 1000), (64, 0), (2, 95)]),
    (64, 48, 16, 8, None, [(200, 13), (33, 190)]), (80, 64, 5, 4, None, [(77, 0), (70, 26)]), (16, 16, 3, 32, None, [(150, 0), (95, 96)]),
    (48, 32, 1, 48, None, [(400, 5)]), (96, 96, 130, 16, None, [(3, 700), (2, 0)]), (256, 256, 9, 64, None, [(130, 62), (65, 64)]),
    (192, 176, 40, 128, None, [(66, 190)]), (144, 112, 7, 16, 33, [(200, 300), (96, 0)]), (256, 192, 4, 32, 150, [(290, 410), (96, 96)]),
    (64, 64, 12, 16, 1, [(100, 37)]), (112, 80, 17, 12, None, [(96, 0), (97, 95)])]


@pytest.mark.parametrize("sinks", [False, True])
@pytest.mark.parametrize("shape", LATENT_TC5)
def test_latent_attention_on_tcgen05_against_the_exact_kernel(shape, sinks):
    """Row sizes and value columns off the 64-column blocks, groups of 1 to 130 heads, both key tiles, portions on both
    sides of a tile's border and behind hundreds of cached rows, windows whose earlier pages are gone (and hold NaN), loud
    keys in the first and last rows; a single row is left to the decode kernel."""
    D, DV, H, page, window, portions = shape
    rt = Runtime(torch.device("cuda"), torch.bfloat16)
    g = torch.Generator().manual_seed(D + H)
    lens, held = [n for n, _ in portions], [p for _, p in portions]
    kv = [n + p for n, p in portions]
    T = sum(lens)
    width = max(-(-k // page) for k in kv)
    per = [-(-k // page) for k in kv]
    order = torch.randperm(sum(per) + 2, generator=g).tolist()
    table = torch.full((len(kv) + 1, width), -1, dtype=torch.int32)
    pages = torch.randn(sum(per) + 2, 1, page, D, generator=g)
    slots = [len(kv) - i for i in range(len(kv))]
    at = 0
    for slot, n, k, p in zip(slots, per, kv, held):
        mine = order[at:at + n]
        at += n
        table[slot, :n] = torch.tensor(mine, dtype=torch.int32)
        for key in (0, k - 1, max(0, k - 97)):
            pages[mine[key // page], 0, key % page] *= 3.0
        pages[mine[-1], 0, (k - 1) % page + 1:] = float("nan")             # behind the last key
        if window is not None:
            for blk in range(max(0, p - window + 1) // page):              # given back: nobody may read them
                pages[mine[blk]] = float("nan")
                table[slot, blk] = -1
    q = (torch.randn(T, H * D, generator=g) * 2).to(torch.bfloat16).cuda()
    pages, table = pages.to(torch.bfloat16).cuda(), table.cuda()
    sink = (torch.randn(H, generator=g) * 4).cuda() if sinks else None
    gate = torch.rand(T, H, generator=g).cuda() if sinks else None
    starts = [sum(lens[:i]) for i in range(len(lens))]
    positions = [p + i for n, p in portions for i in range(n)]
    seq_of = [i for i, n in enumerate(lens) for _ in range(n)]
    ctx = ctx_of(rt, positions, seq_of, slots, starts, lens, kv)
    exact = torch.zeros(T, H * D, dtype=torch.bfloat16, device="cuda")
    ops.attention_generic(exact, q, ctx.positions, ctx.seq_of_token, ctx.seq_slot, table, pages, pages, T, H, 1, D,
                          ops.visible_reach(window, None), D ** -0.5, ctx.status, sink=sink, gate=gate)
    out = torch.full((T, H * D), 7.0, dtype=torch.bfloat16, device="cuda")
    ops.attention_latent_tcgen05(out, q, ctx.seq_q_start, ctx.seq_q_len, ctx.seq_kv_len, ctx.seq_slot, table, pages, len(kv), max(lens),
                                 H, 1, D, DV, ops.visible_reach(window, None), D ** -0.5, True, ctx.status, sink=sink, gate=gate)
    assert int(ctx.status) == 0
    got, want = out.float().cpu().view(T, H, D), exact.float().cpu().view(T, H, D)
    for n, at in zip(lens, starts):
        rows = slice(at, at + n)
        if n == 1:
            assert bool((got[rows] == 7.0).all())
            continue
        assert bool((got[rows][:, :, DV:] == 7.0).all())                   # columns that are no values are not written
        close(got[rows][:, :, :DV], want[rows][:, :, :DV], torch.bfloat16, f"portion of {n}", bf16=1.5e-2)


MAMBA_SHAPES = [  # hidden, heads, value size, state, groups, taps, norm parts
    (48, 4, 16, 16, 2, 4, 1), (40, 3, 6, 10, 3, 6, 2), (36, 4, 5, 7, 1, 1, 5), (64, 2, 24, 32, 1, 3, 3), (40, 1, 24, 16, 1, 2, 1),
    (96, 4, 48, 32, 2, 4, 2), (64, 2, 64, 128, 1, 4, 1), (64, 6, 64, 64, 3, 4, 2), (64, 4, 32, 48, 2, 5, 4), (40, 2, 40, 96, 1, 4, 8),
    (48, 8, 64, 16, 2, 4, 4), (48, 2, 112, 64, 1, 4, 1), (64, 3, 64, 256, 1, 4, 3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MAMBA_SHAPES)
def test_state_space_mixer_alone(dtype, shape):
    """Convolution with a bias, step sizes, decays, the skip, shared groups, the gate and the norm of parts; two requests
    in slots of their own, cut into steps of 1 to 150 rows."""
    hidden, heads, vdim, state, groups, taps, parts = shape
    rt = Runtime(torch.device("cuda"), dtype)
    layer = mamba(heads, vdim, state, groups, taps, parts)
    mixer = mixer_of(rt, hidden, layer)
    w = filled(mixer, 12, 0.3)
    g = torch.Generator().manual_seed(5)
    set_weight(mixer, w, "conv", torch.randn(w["conv"].shape, generator=g) * 0.6)
    set_weight(mixer, w, "A_log", torch.randn(heads, generator=g))
    set_weight(mixer, w, "dt_bias", torch.randn(heads, generator=g) - 1.0)
    set_weight(mixer, w, "D", torch.randn(heads, generator=g))
    wd = {k: v.double() for k, v in named(w).items()}
    run_state_mixer(rt, mixer, hidden, lambda h, pos: plain.mixer_mamba2(h, wd, "p.", layer["mixer"], 1e-5))


def stored_as(dtype):
    """The rounding of rows kept in ``dtype``, for the plain mixer: where sums over keys cancel (a state of one loud token, a
    step size of a hundred) rounding the rows alone moves an output by several per cent."""
    return (lambda t: t) if dtype == torch.float32 else (lambda t: t.to(torch.bfloat16).double())


def walk_by_hand(x, b, c, dt, rate, skip, S):
    """The recurrence from a given state, in float64: (y, the state behind the last token)."""
    y = torch.empty_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(-rate * dt[t])[:, None, None] * S + (dt[t][:, None] * b[t])[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, c[t]) + skip[:, None] * x[t]
    return y, S


@pytest.mark.parametrize("heads,groups,state,vdim,slice_dim", [
    (4, 2, 16, 16, 16), (3, 1, 16, 64, 64), (2, 2, 32, 32, 32), (4, 1, 32, 48, 16), (6, 3, 64, 64, 64), (2, 1, 64, 64, 32), (3, 3, 64, 32, 16),
    (2, 1, 128, 64, 64), (4, 2, 128, 128, 64), (2, 1, 128, 96, 32), (1, 1, 128, 16, 16), (2, 1, 256, 64, 64), (2, 2, 256, 32, 32)])
def test_recurrence_in_chunks_on_the_tensor_cores(heads, groups, state, vdim, slice_dim):
    """Six requests side by side of 1 to 200 tokens (chunk borders on both sides), states that are not zero at the start,
    fast and slow heads, slots in another order than the requests; outputs and states against a walk in float64, to far
    below what a bfloat16 rounding of state, decays or step sizes would leave."""
    g = torch.Generator().manual_seed(state + vdim)
    lens = [64, 1, 65, 200, 63, 2]
    slots = [3, 0, 6, 2, 5, 1]
    T, N, channels = sum(lens), state, heads * vdim + 2 * groups * state
    rows = torch.randn(T, channels, generator=g).to(torch.bfloat16)
    pre = torch.randn(T, heads, generator=g)
    rate_log, bias, skip = (torch.randn(heads, generator=g) * 1.5 - off for off in (1.0, 1.0, 0.0))
    init = torch.randn(7, heads * N * vdim + 6, generator=g)
    st = init.cuda().clone()
    out = torch.full((T, heads * vdim), float("nan"), device="cuda")
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")     # noqa: E731
    starts = [sum(lens[:i]) for i in range(len(lens))]
    dev = rows.cuda()
    hv, gn = heads * vdim, groups * N
    args = (dev[:, hv + gn:], dev[:, hv:hv + gn], dev[:, :hv], pre.cuda(), rate_log.cuda(), bias.cuda(), skip.cuda())
    ops.state_space_chunks(out, *args, st, i32(slots), i32(starts), i32(lens), len(lens), heads, N, vdim, heads // groups, True, slice_dim=slice_dim)
    kept = init.cuda().clone()
    again = torch.empty_like(out)
    ops.state_space_chunks(again, *args, kept, i32(slots), i32(starts), i32(lens), len(lens), heads, N, vdim, heads // groups, False, slice_dim=slice_dim)
    assert torch.equal(again, out) and torch.equal(kept.cpu(), init)              # without the write the slots stay as they were
    d = rows.double()
    x, b, c = d[:, :hv].view(T, heads, vdim), d[:, hv:hv + gn].view(T, groups, N), d[:, hv + gn:].view(T, groups, N)
    b, c = (t.repeat_interleave(heads // groups, dim=1) for t in (b, c))
    dt = plain.softplus(pre.double() + bias.double())
    got, got_state = out.cpu().double(), st.cpu().double()
    for n, slot, at in zip(lens, slots, starts):
        one = slice(at, at + n)
        S0 = init[slot, :heads * N * vdim].double().view(heads, N, vdim)
        y, S = walk_by_hand(x[one], b[one], c[one], dt[one], torch.exp(rate_log.double()), skip.double(), S0)
        for h in range(heads):
            scale = float(y[:, h].abs().max())
            assert float((got[one].view(n, heads, vdim)[:, h] - y[:, h]).abs().max()) <= 1e-4 * scale, (n, h)
            state_got = got_state[slot, :heads * N * vdim].view(heads, N, vdim)[h]
            assert float((state_got - S[h]).abs().max()) <= 1e-4 * float(S[h].abs().max()), (n, h)
        assert torch.equal(got_state[slot, heads * N * vdim:], init[slot, heads * N * vdim:].double())     # what lies behind the heads
    assert torch.equal(got_state[4], init[4].double())                           # nobody's slot


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("vdim,state", [(16, 16), (64, 128), (64, 64), (32, 32)])
@pytest.mark.parametrize("loud_row", [0, 3, 149])
def test_state_keeps_one_token_from_far_back(dtype, vdim, state, loud_row):
    """Slow decays, no skip and one loud token: hundreds of tokens later the outputs still consist mostly of what that
    token left in the state, through cuts into steps of 1 to 150 tokens.  A state that is lost, zeroed or taken from
    another slot on the way shows at once."""
    rt = Runtime(torch.device("cuda"), dtype)
    hidden, heads = 48, 2
    layer = mamba(heads, vdim, state, 1, 4, 1)
    mixer = mixer_of(rt, hidden, layer)
    w = filled(mixer, 22, 0.3)
    set_weight(mixer, w, "A_log", torch.full((heads,), -7.0))           # 0.999 per unit of step size
    set_weight(mixer, w, "dt_bias", torch.full((heads,), -1.0))
    set_weight(mixer, w, "D", torch.zeros(heads))
    wd = {k: v.double() for k, v in named(w).items()}
    run_state_mixer(rt, mixer, hidden, lambda h, pos: plain.mixer_mamba2(h, wd, "p.", layer["mixer"], 1e-5, stored_as(dtype)),
                    loud_row=loud_row, bf16=1.5e-2)


@pytest.mark.parametrize("channels,taps,with_bias", [(256, 4, True), (1032, 3, True), (64, 2, False), (40, 4, True), (2056, 4, False), (48, 1, True), (20, 4, True)])
@pytest.mark.parametrize("out_dtype", DTYPES)
def test_convolution_over_mixed_rows(channels, taps, with_bias, out_dtype):
    """bfloat16 rows of nine requests of 1 to 70 rows with padding rows in between, every request with inputs kept from
    before; single rows move their state on.  Channels in eights (16-byte accesses) and not."""
    g = torch.Generator().manual_seed(channels + taps)
    lens = [1, 2, 3, 17, 1, 70, 4, 33, 1]
    rows, seq_of, starts = [], [], []
    for i, n in enumerate(lens):
        starts.append(len(seq_of))
        seq_of += [i] * n + [-1] * (i % 3)
    T = len(seq_of)
    x = torch.randn(T, channels + 8, generator=g).to(torch.bfloat16)
    w, bias = torch.randn(channels, taps, generator=g), torch.randn(channels, generator=g) if with_bias else None
    slots = [8, 3, 5, 0, 7, 1, 6, 2, 4]
    state = torch.randn(9, 5 + channels * (taps - 1), generator=g)
    st = state.cuda().clone()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")     # noqa: E731
    out = torch.full((T, channels), float("nan"), dtype=out_dtype, device="cuda")
    dev = x.cuda()
    ops.short_conv(out, dev[:, 8:], w.cuda(), st, 5, i32(seq_of), i32(slots), i32(starts), T, move_single=i32(lens),
                   bias=None if bias is None else bias.cuda())
    got, after = out.float().cpu(), st.cpu()
    for n, slot, at in zip(lens, slots, starts):
        kept = state[slot, 5:].view(channels, taps - 1).T.double()
        seq = torch.cat([kept, x[at:at + n, 8:].double()])
        y = sum(seq[j:j + n] * w[:, j].double() for j in range(taps)) + (0 if bias is None else bias.double())
        close(got[at:at + n], plain.silu(y).float(), out_dtype, f"request of {n} rows", bf16=5e-3)
        want = seq[1:].T.reshape(-1).float() if n == 1 and taps > 1 else state[slot, 5:]
        assert torch.equal(after[slot, 5:], want) and torch.equal(after[slot, :5], state[slot, :5])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [2, 4, 6])
def test_convolution_at_the_first_tokens_and_across_steps(dtype, taps):
    """Weights so large at the oldest tap that a row missing ahead of a step, or one too many at a request's start, moves
    the output by its size: requests of fewer rows than taps, single rows first, steps shorter than the taps."""
    rt = Runtime(torch.device("cuda"), dtype)
    hidden = 32
    layer = mamba(2, 16, 16, 1, taps, 1)
    mixer = mixer_of(rt, hidden, layer)
    w = filled(mixer, 31, 0.3)
    conv = 0.2 * torch.randn(w["conv"].shape, generator=torch.Generator().manual_seed(6))
    conv[:, 0] *= 8.0
    set_weight(mixer, w, "conv", conv)
    set_weight(mixer, w, "conv.b", 0.5 * torch.randn(w["conv.b"].shape, generator=torch.Generator().manual_seed(7)))
    wd = {k: v.double() for k, v in named(w).items()}
    run = lambda h, pos: plain.mixer_mamba2(h, wd, "p.", layer["mixer"], 1e-5)      # noqa: E731
    for plan in (((1, 1), (1, 0), (1, 1), (2, 1), (1, 0), (3, 2)), ((2, 1), (2, 3), (2, 1), (3, 0)), ((9, 5),), ((1, 5),) + ((1, 0),) * 8):
        run_state_mixer(rt, mixer, hidden, run, lengths=(9, 5), plan=plan)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("extreme", ["fast", "slow", "large"])
def test_decays_at_their_extremes(dtype, extreme):
    """Decays that underflow to zero within a token, that are one to many digits, and step sizes of a hundred: no value
    that is not finite, and the plain outputs."""
    rt = Runtime(torch.device("cuda"), dtype)
    hidden, heads = 48, 2
    layer = mamba(heads, 64, 64, 1, 4, 1)
    mixer = mixer_of(rt, hidden, layer)
    w = filled(mixer, 41, 0.3)
    a, b = {"fast": (5.0, 3.0), "slow": (-12.0, -6.0), "large": (-1.0, 100.0)}[extreme]
    set_weight(mixer, w, "A_log", torch.tensor([a, a - 2.0])); set_weight(mixer, w, "dt_bias", torch.tensor([b, b + 0.5]))
    wd = {k: v.double() for k, v in named(w).items()}
    run_state_mixer(rt, mixer, hidden, lambda h, pos: plain.mixer_mamba2(h, wd, "p.", layer["mixer"], 1e-5, stored_as(dtype)),
                    bf16=1.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,experts,top,ff,scale,groups", [
    (64, 8, 3, 40, 2.0, (4, 2)), (40, 5, 1, 20, 1.0, None), (36, 6, 2, 9, 0.5, (3, 1)), (128, 12, 4, 88, 1.5, (6, 3)), (48, 4, 4, 16, 1.0, (2, 2)),
    (64, 72, 6, 16, 2.5, (8, 3)), (48, 40, 8, 24, 1.0, (20, 6)), (48, 1, 1, 16, 1.7, (1, 1))])
def test_experts_within_groups_alone(dtype, hidden, experts, top, ff, scale, groups):
    """Scores over all experts, the best groups by their best score, the choice inside them, weights renormalised over
    the chosen ones; rows whose choice no rounding can turn."""
    rt = Runtime(torch.device("cuda"), dtype)
    mlp = moe(experts, top, ff, scale, groups)
    typed, layer = typed_layer(hidden, mamba(1, 8, 8, 1, 2, 1, mlp))
    part = build_part("feed_forward", feed_forward_spec(typed, layer.mlp), rt)
    w = fill(part, 14, 0.3)
    g = torch.Generator().manual_seed(2)
    rows = 61
    h = torch.randn(rows, hidden, generator=g).to(dtype)
    w["router"] = (torch.randn(experts, hidden, generator=g) * 0.4).to(torch.bfloat16).float()
    part.w_router.copy_(w["router"])
    wd = {k: v.double() for k, v in named(w).items()}
    want = plain.mixture(h.double(), wd, "p.", mlp).float()
    chosen_want, weight_want = plain.route(h.double(), wd, "p.", mlp["router"])
    # rows that are far enough from another choice: of groups, and of experts inside the kept groups
    s = torch.softmax(h.double() @ wd["p.router"].T, -1)
    sure = torch.ones(rows, dtype=torch.bool)
    inside = s
    if groups is not None:
        best = s.view(rows, groups[0], -1).max(-1).values.sort(-1, descending=True).values
        if groups[1] < groups[0]:
            sure &= best[:, groups[1] - 1] > 1.02 * best[:, groups[1]]
        kept = s.view(rows, groups[0], -1).max(-1).values >= best[:, groups[1] - 1:groups[1]]
        inside = s * kept.repeat_interleave(experts // groups[0], dim=1)
    ranked = inside.sort(-1, descending=True).values
    if top < experts:
        sure &= ranked[:, top - 1] > 1.02 * ranked[:, top]
    assert int(sure.sum()) >= rows // 2
    ctx = ctx_of(rt, list(range(rows)), [0] * rows, [0], [0], [rows], [rows])
    chosen, weight, _ = part.route(ctx, h.cuda())
    assert torch.equal(chosen.cpu().long().sort(-1).values[sure], chosen_want.sort(-1).values[sure])
    lookup = torch.zeros(rows, experts, dtype=torch.float64).scatter_(1, chosen_want, weight_want)
    close(weight.cpu()[sure], torch.gather(lookup, 1, chosen.cpu().long())[sure].float(), torch.float32, "weights of the chosen",
          f32=2e-2 if dtype == torch.bfloat16 else 1e-5)
    close(weight.sum(-1).cpu(), torch.full((rows,), scale), torch.float32, "sums of the weights", f32=1e-5)
    if groups is not None and groups[1] < groups[0] and top > 1:
        free, _ = plain.route(h.double(), wd, "p.", {**mlp["router"], "groups": None})
        assert bool((free.sort(-1).values != chosen_want.sort(-1).values).any())      # the groups are felt
    for n in (rows, 1):                                            # sorted by expert (bfloat16, several rows), and pair by pair
        one = ctx_of(rt, list(range(n)), [0] * n, [0], [0], [n], [n])
        got = dense_delta(one, part.forward(one, h[:n].cuda()), dtype).float().cpu()
        close(got[sure[:n]], want[:n][sure[:n]], dtype, f"routed feed-forward, {n} rows") if bool(sure[:n].any()) else None


@pytest.mark.parametrize("dtype", DTYPES)
def test_equal_scores_choose_the_lowest_index(dtype):
    """A router of zeros: every score is equal, the first groups and the first experts in them are chosen, in order."""
    rt = Runtime(torch.device("cuda"), dtype)
    typed, layer = typed_layer(32, mamba(1, 8, 8, 1, 2, 1, moe(72, 5, 16, 2.0, (36, 4))))
    part = build_part("feed_forward", feed_forward_spec(typed, layer.mlp), rt)
    fill(part, 14, 0.3)
    part.w_router.zero_()
    ctx = ctx_of(rt, [0, 1], [0, 0], [0], [0], [2], [2])
    chosen, weight, _ = part.route(ctx, torch.randn(2, 32).to(dtype).cuda())
    assert chosen.tolist() == [[0, 1, 2, 3, 4]] * 2
    close(weight.cpu(), torch.full((2, 5), 0.4), torch.float32, "weights", f32=1e-6)


# ---------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------
def settle_router(folder):
    """For bfloat16 runs: a router whose choice no rounding can turn.  Channel 0 of the stream is made a constant (every
    embedding row has the same value there and no sub-layer writes it), and the router's column that reads it ranks a
    layer's experts far apart, in an order of the layer's own; the rest of the router still moves the weights with the
    token.  (The choice per token is what the float32 runs, whose routers are as random as every other matrix, and the
    test of the part alone check.)"""
    from safetensors.torch import load_file, save_file
    t = load_file(str(folder / "model.safetensors"))
    t["embed"][:, 0] = 2.0
    for name in sorted(t):
        if name.endswith((".mix.o", ".mlp.down")) or (".mlp.e" in name and name.endswith(".down")):
            t[name][0, :] = 0.0
        if name.endswith(".mlp.router"):
            g = torch.Generator().manual_seed(len(name) + t[name].shape[0])
            t[name] = (t[name].float() * 0.25).to(t[name].dtype)
            t[name][:, 0] = (torch.randperm(t[name].shape[0], generator=g).float() * 0.8).to(t[name].dtype)
    save_file({k: v.contiguous() for k, v in t.items()}, str(folder / "model.safetensors"), metadata={"format": "pt"})
    return folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """(name, dtype) -> model folder; the bfloat16 runs get a copy whose routers are settled."""
    tmp = tmp_path_factory.mktemp("bavetar")
    out = {}
    for name, cfg in BAVETAR_CONFIGS.items():
        out[name, "float32"] = tw.write_random_model(tmp / name, cfg, seed=BAVETAR_SEEDS[name], std=BAVETAR_STD[name])
        out[name, "bfloat16"] = settle_router(tw.write_random_model(tmp / f"{name}_settled", cfg, seed=BAVETAR_SEEDS[name], std=BAVETAR_STD[name]))
    return out


LENGTHS = [70, 1, 45, 100, 2, 33, 64, 129]


def requests_for(name):
    return {f"r{i}": random_tokens(BAVETAR_CONFIGS[name]["vocab"], n, 20 + i) for i, n in enumerate(LENGTHS)}


@pytest.fixture(scope="module")
def plain_rows(folders):
    return {key: {rid: plain.logits_of(folder, t).numpy() for rid, t in requests_for(key[0]).items()}
            for key, folder in folders.items()}


def moved_weights(folder, seed):
    """The plain model with every matrix element moved by a relative 2^-8 times a normal draw."""
    config, weights = plain.read_folder(folder, torch.float64)
    g = torch.Generator().manual_seed(seed)
    return config, {k: v * (1 + 2.0 ** -8 * torch.randn(v.shape, generator=g, dtype=torch.float64)) if v.dim() == 2 else v
                    for k, v in weights.items()}


def lost_rows(folder, dtype, tokens, want, seed):
    """What the arithmetic alone does to each row: the plain model in float32, or with perturbed matrices, against itself."""
    low = plain.logits_of(folder, tokens, torch.float32) if dtype == "float32" else plain.forward(*moved_weights(folder, seed), tokens).float()
    return [row_error(low[p].numpy(), want[p]) for p in range(len(tokens))]


@pytest.fixture(scope="module")
def noise(folders, plain_rows):
    return {(name, dtype, rid): lost_rows(folder, dtype, t, plain_rows[name, dtype][rid], 99)
            for (name, dtype), folder in folders.items() for rid, t in requests_for(name).items()}


def compare(rows, want, dtype, what, lost):
    """Every logits row against the plain one (float64).  float32: every row within 5e-5 of its spread plus four
    times what the plain implementation loses at that row when it runs in float32 itself.  bfloat16: the median within
    4 %, at most five rows in a hundred beyond 6 % plus three times what a perturbation of bfloat16's size does to that
    row of the plain implementation, none that is not finite.  A lost state, a key that is missed or a wrong page moves
    rows by their whole size."""
    errors, over = [], []
    for (rid, p), row in rows.items():
        err = row_error(row, want[rid][p])
        assert np.isfinite(row).all(), f"{what}: {rid}[{p}] is not finite"
        if dtype == "float32":
            assert err <= 5e-5 + 4 * lost[rid][p], f"{what}: {rid}[{p}] differs by {err:.3g} of the row's spread (float32 alone: {lost[rid][p]:.3g})"
        elif err > 6e-2 + 3 * lost[rid][p]:
            over.append((rid, p, round(err, 3)))
        errors.append(err)
    if dtype == "bfloat16":
        assert float(np.median(errors)) <= 4e-2, f"{what}: the median row differs by {float(np.median(errors)):.3g}"
        assert len(over) <= max(2, 5 * len(errors) // 100), f"{what}: {len(over)} of {len(errors)} rows are far off: {over[:8]}"


SCHEDULES = {
    "whole": schedule_whole,
    "tail": schedule_tail,
    "portions": schedule_portions,
    "pairs": lambda r: schedule_portions({k: v for k, v in r.items() if len(v) <= 70}, sizes=(2,)),
    "one_by_one": lambda r: schedule_portions({k: v for k, v in r.items() if len(v) <= 70}, sizes=(1,)),
    "mixed": lambda r: schedule_mixed(r, live=4, seed=1),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(BAVETAR_CONFIGS))
def test_every_cutting_gives_the_plain_logits(name, dtype, folders, plain_rows, noise, tmp_path):
    """Whole prompts; most of a prompt and its last 32 tokens one by one; portions down to two tokens; token by
    token from the first; four live requests in mixed batches with so few pages and slots that both are used
    again (freed pages are filled with NaN first)."""
    reqs = requests_for(name)
    for kind, make in SCHEDULES.items():
        steps = make(reqs)
        rows = replay_in_process(folders[name, dtype], dtype, steps, tmp_path / kind, block_size=BAVETAR_PAGE[name],
                                 max_tokens=max_live_tokens(steps))
        assert rows, kind
        compare(rows, plain_rows[name, dtype], dtype, f"{name} {kind}", {rid: noise[name, dtype, rid] for rid in reqs})


@pytest.mark.parametrize("name", ["A", "C"])
def test_batches_and_cuts_do_not_change_a_request(name, folders, tmp_path):
    """float32: a request's logits in a mixed batch, or cut into portions, equal those it gets alone, to rounding."""
    reqs = requests_for(name)
    folder = folders[name, "float32"]
    alone = replay_in_process(folder, "float32", schedule_whole(reqs), tmp_path / "alone", block_size=8)
    for kind, steps in (("mixed", schedule_mixed(reqs, live=4, seed=3)), ("portions", schedule_portions(reqs))):
        got = replay_in_process(folder, "float32", steps, tmp_path / kind, block_size=8)
        worst = max(float(np.abs(row - alone[key]).max() / np.abs(alone[key]).max()) for key, row in got.items())
        assert worst <= 1e-4, (kind, worst)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_used_again(dtype, folders):
    """One request slot and barely enough pages: each request gets the slot and the pages its predecessor gave back,
    with the predecessor's states and latents still in them (the manager zeroes the states at admission)."""
    from tessweave_engine_b200.engine.runner import ModelRunner, StepEntry
    name = "A"
    folder = folders[name, dtype]
    model = tw.load_model(folder, dtype, "cuda")
    cache = tw.CacheManager(model.cache_needs(), BAVETAR_PAGE[name], 9, 1, 72, model.runtime.dtype, model.runtime.device,
                            prefix_cache=False)
    runner = ModelRunner(model, cache, 72, 1, cuda_graphs=False)
    for i, n in enumerate([70, 64, 3, 71]):
        tokens = random_tokens(BAVETAR_CONFIGS[name]["vocab"], n, 40 + i)
        lease = cache.admit(None)
        assert lease.slot == 0
        cut = max(1, n // 2)
        cache.ensure(lease, cut)
        runner.step([StepEntry(lease.slot, tokens[:cut], 0, [])])
        cache.ensure(lease, n)
        got = runner.step([StepEntry(lease.slot, tokens[cut:], cut, list(range(n - cut)))]).cpu().numpy()
        runner.check_status()
        cache.release(lease)
        cache.check_invariants()
        want = plain.logits_of(folder, tokens).numpy()
        compare({("r", cut + k): got[k] for k in range(n - cut)}, {"r": want}, dtype, f"request {i} in a used slot",
                {"r": lost_rows(folder, dtype, tokens, want, 96)})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, folders, tmp_path):
    """A short prompt and 300 tokens one by one: decode attention over many pages, the states carry everything else."""
    name = "C"
    toks = random_tokens(BAVETAR_CONFIGS[name]["vocab"], 310, 77)
    rows = replay_in_process(folders[name, dtype], dtype, schedule_tail({"long": toks}, tail=300), tmp_path / "out",
                             block_size=BAVETAR_PAGE[name], max_tokens=384)
    want = plain.logits_of(folders[name, dtype], toks).numpy()
    compare(rows, {"long": want}, dtype, "long decoding", {"long": lost_rows(folders[name, dtype], dtype, toks, want, 97)})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_of_hundreds_of_tokens(dtype, tmp_path):
    """Prompts of 420 and 190 tokens on pages of 16: whole, with the last 40 tokens one by one, and in mixed batches."""
    folder = tw.write_random_model(tmp_path / "model", BAVETAR_E, seed=31, std=0.1)
    if dtype == "bfloat16":
        settle_router(folder)
    vocab = BAVETAR_E["vocab"]
    reqs = {"long": random_tokens(vocab, 420, 5), "mid": random_tokens(vocab, 190, 6), "short": random_tokens(vocab, 37, 7)}
    want = {rid: plain.logits_of(folder, t).numpy() for rid, t in reqs.items()}
    lost = {rid: lost_rows(folder, dtype, t, want[rid], 98) for rid, t in reqs.items()}
    for kind, steps in (("whole", schedule_whole(reqs)), ("tail", schedule_tail(reqs, tail=40)),
                        ("mixed", schedule_mixed(reqs, live=3, seed=2, prefill=(33, 2, 70, 5, 128, 16)))):
        rows = replay_in_process(folder, dtype, steps, tmp_path / kind, block_size=16, max_tokens=max_live_tokens(steps))
        compare(rows, want, dtype, f"E {kind}", lost)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_engine(name, dtype, folders):
    """``generate`` (scheduler, continuous batching, CUDA graphs, look-ahead) against the plain greedy loop;
    every chosen token must be the plain implementation's best on that path, or nearly."""
    prompts = [random_tokens(BAVETAR_CONFIGS[name]["vocab"], n, 60 + n) for n in (21, 5, 40)]
    model = tw.load_model(folders[name, dtype], dtype, "cuda")
    out = tw.generate(model, prompts, max_tokens=12, ignore_eos=True,
                      engine_config=tw.EngineConfig(block_size=BAVETAR_PAGE[name], kv_blocks=40, max_context=128, max_active=2,
                                                    prefill_chunk=16))
    config, weights = plain.read_folder(folders[name, dtype], torch.float64)
    for p, o in zip(prompts, out):
        assert len(o) == 12
        logits = plain.forward(config, weights, p + o).float()
        for i, t in enumerate(o):
            row = logits[len(p) + i - 1]
            gap, spread = float(row.max() - row[t]), float(row.std())
            assert gap <= (1e-4 if dtype == "float32" else 0.15) * spread, f"token {i} lies {gap:.3g} below the best (spread {spread:.3g})"

"""The Varivik decoder in the engine against the plain implementation (tests/plain_varivik.py): every mechanism alone,
then whole models under every way of cutting and batching the work, in float32 and bfloat16.  The tiny models and their
weights are made here."""
import numpy as np
import pytest
import torch

import plain_varivik as plain
import tessweave_engine_b200 as tw
from helpers import (max_live_tokens, random_tokens, replay_in_process, schedule_mixed, schedule_portions, schedule_tail,
                     schedule_whole)
from test_gpu_linurax import close, ctx_of, fill
from test_gpu_nufatar import filled, run_attention, set_weight
from test_gpu_sapatar import named, row_error, step_ctx
from tessweave_engine_b200.config.varivik_config import VarivikConfig
from tessweave_engine_b200.csrc import ops
from tessweave_engine_b200.csrc.ops import SplitSum
from tessweave_engine_b200.models.varivik import attention_spec, feed_forward_spec
from tessweave_engine_b200.parts import PartSpec, Runtime, build_part, dense_delta
from tiny_varivik import (VARIVIK_CONFIGS, VARIVIK_E, VARIVIK_PAGE, VARIVIK_SEEDS, VARIVIK_STD, attention, bands, dense, moe, rot)

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def typed_layer(width, layer, eps=1e-5):
    """The typed configuration of a model of one layer, and that layer."""
    typed = VarivikConfig.from_dict({"vocab": 8, "width": width, "norm": {"eps": eps}, "layers": [layer]})
    return typed, typed.layers[0]


def mixer_of(rt, width, layer, first=True):
    typed, one = typed_layer(width, layer)
    return build_part("mixer", attention_spec(typed, one.mixer, first), rt)


def doubles(w):
    return {k: v.double() for k, v in named(w).items()}


# ---------------------------------------------------------------------------
# the pass over the projected rows
# ---------------------------------------------------------------------------
PREPARE = [  # heads, kv heads, key size, value size, rotated, neighbours?, slices (0: rows), page
    (4, 2, 16, 32, 8, True, 0, 8), (3, 1, 7, 5, 6, True, 0, 4), (8, 2, 64, 32, 32, True, 5, 16), (4, 4, 24, 24, 24, True, 3, 4),
    (6, 3, 32, 16, 16, False, 2, 8), (2, 1, 128, 64, 128, True, 12, 16), (5, 5, 8, 8, 0, True, 1, 2), (2, 2, 20, 12, 10, True, 4, 8)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("role", ["none", "leave", "mix"])
@pytest.mark.parametrize("shape", PREPARE)
def test_rotation_blend_store_and_gates_in_one_pass(dtype, role, shape):
    """q turned by its position into rows of its own; k turned, and v (blended with kept values where asked), in their
    places of the pages and nowhere else; the gates' sigmoids; from rows and from the slices of a split product."""
    H, G, D, Dv, dims, neighbours, nslices, page = shape
    rt = Runtime(torch.device("cuda"), dtype)
    g = torch.Generator().manual_seed(D + Dv)
    positions = [0, 1, 2, 70, 5, 6, 0]
    n, used = len(positions), H * D + G * (D + Dv) + H
    width = -(-used // 8) * 8
    theta = 300.0
    plan = build_part("position", PartSpec("rope_interleaved" if neighbours else "rope", {
        "theta": theta, "dims": dims, **({"bands": bands(4.0, 1.0, 4.0, 64)} if neighbours else {})}), rt).rotary_plan(D)
    if nslices:
        slices = torch.randn(nslices, n, width, generator=g)
        slices[:, :, used:] = float("nan")              # columns nobody may read
        x, rows = slices.sum(0).double(), SplitSum(slices.cuda())
    else:
        x = torch.randn(n, width, generator=g).to(dtype)
        x[:, used:] = float("nan")
        x, rows = x.double(), x.cuda()
    kept = torch.randn(n, G * Dv, generator=g).to(dtype)
    lam = torch.tensor([0.3])
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")     # noqa: E731
    seq = [0, 0, 0, 1, 2, 2, -1]                        # the last row is padding
    table = torch.full((3, 40), -1, dtype=torch.int32)
    pages = 0
    for s, p in ((0, 0), (0, 1), (0, 2), (1, 70), (2, 5), (2, 6)):
        if table[s, p // page] < 0:
            table[s, p // page] = 2 * pages + 1
            pages += 1
    k_pages = torch.full((2 * pages + 1, G, page, D), 7.0, dtype=dtype, device="cuda")
    v_pages = torch.full((2 * pages + 1, G, page, Dv), 7.0, dtype=dtype, device="cuda")
    q_out = torch.full((n, H * D), 7.0, dtype=dtype, device="cuda")
    gate = torch.full((n, H), 7.0, device="cuda")
    left = torch.full((n, G * Dv), 7.0, dtype=dtype, device="cuda")
    status = i32([0])
    more = {"leave": {"leave_values": left}, "mix": {"mix_values": kept.cuda(), "mix_weight": lam.cuda()}, "none": {}}[role]
    ops.attention_prepare(q_out, rows, n, H, G, D, Dv, i32(positions), i32(seq), i32([0, 1, 2]), table.cuda(), k_pages, v_pages,
                          True, status, rot_dims=plan.rot_dims, inv_freq=plan.inv_freq, interleaved=plan.interleaved, gate=gate, **more)
    assert int(status) == 0
    q, k, v, z = x[:, :H * D].reshape(n, H, D), x[:, H * D:H * D + G * D].reshape(n, G, D), \
        x[:, H * D + G * D:used - H].reshape(n, G, Dv), x[:, used - H:used]
    pos = torch.tensor(positions)
    if neighbours:
        rates = plain.turning_rates(dims, theta, bands(4.0, 1.0, 4.0, 64))
        q, k = plain.rotate_neighbours(q, pos, dims, rates), plain.rotate_neighbours(k, pos, dims, rates)
    else:
        order = [j for i in range(dims // 2) for j in (i, i + dims // 2)] + list(range(dims, D))
        back = torch.argsort(torch.tensor(order))
        rates = plain.turning_rates(dims, theta, None)
        q, k = (plain.rotate_neighbours(t[..., order], pos, dims, rates)[..., back] for t in (q, k))
    if role == "mix":
        v = plain.mix_values(v, kept.double().reshape(n, G, Dv), 0.3)
    close(q_out[:6].double().cpu(), q.reshape(n, -1)[:6], dtype, "q", f32=1e-5, bf16=1e-2)
    close(gate[:6].double().cpu(), torch.sigmoid(z)[:6], torch.float32, "gates")
    if role == "leave":
        close(left[:6].double().cpu(), v.reshape(n, -1)[:6], dtype, "kept values", bf16=1e-2)
    touched_k, touched_v = torch.zeros_like(k_pages, dtype=torch.bool), torch.zeros_like(v_pages, dtype=torch.bool)
    for row, (s, p) in enumerate(zip(seq, positions)):
        if s < 0:
            continue
        at = int(table[s, p // page])
        close(k_pages[at, :, p % page].double().cpu(), k[row], dtype, "key", f32=1e-5, bf16=1e-2)
        close(v_pages[at, :, p % page].double().cpu(), v[row], dtype, "value", bf16=1e-2)
        touched_k[at, :, p % page] = True
        touched_v[at, :, p % page] = True
    assert bool((k_pages[~touched_k] == 7).all()) and bool((v_pages[~touched_v] == 7).all())
    table[1] = -1                                      # a page that is not there: the status says so, nothing else is lost
    ops.attention_prepare(q_out, rows, n, H, G, D, Dv, i32(positions), i32(seq), i32([0, 1, 2]), table.cuda(), k_pages, v_pages,
                          True, status, rot_dims=plan.rot_dims, inv_freq=plan.inv_freq, interleaved=plan.interleaved, gate=gate)
    assert int(status) == 2


# ---------------------------------------------------------------------------
# attention alone
# ---------------------------------------------------------------------------
SHAPES = [  # hidden, heads, kv heads, key size, value size, chunk, page, rotation
    (48, 4, 2, 16, 32, 9, 8, rot(8, 1000.0, bands(4.0, 1.0, 4.0, 64))), (40, 3, 1, 12, 20, 5, 4, rot(2, 10.0)),
    (36, 5, 5, 7, 7, 3, 2, rot(6, 50.0)), (64, 6, 3, 64, 64, 40, 16, rot(32, 3e4, bands(8.0, 1.0, 4.0, 64))),
    (64, 4, 2, 64, 32, 50, 16, rot(64, 1e4)), (64, 2, 2, 32, 128, 150, 16, None), (32, 1, 1, 8, 24, 2, 4, rot(8, 20.0)),
    (128, 8, 2, 64, 64, 64, 16, rot(64, 1e6)), (64, 4, 1, 128, 64, 70, 16, rot(64, 1e5)), (96, 4, 1, 80, 48, 33, 16, rot(16, 500.0)),
    (64, 2, 1, 48, 16, None, 8, rot(48, 1e3)), (64, 2, 1, 320, 272, 50, 16, rot(64, 1e4)), (40, 2, 1, 16, 16, 1, 4, rot(16, 30.0)),
    (64, 20, 2, 32, 16, 21, 8, rot(32, 1e3))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_chunked_attention_alone(dtype, shape):
    """Chunks shorter and longer than a page, of one token, and none; keys and values of their own sizes; gates; two
    requests side by side in portions (down to two tokens) and single tokens, pages that a finished chunk gives back on
    the way (and that are filled with NaN then)."""
    hidden, heads, kv, d, dv, chunk, page, turn = shape
    rt = Runtime(torch.device("cuda"), dtype)
    layer = attention(heads, kv, d, dv, 1.5 / d ** 0.5, chunk, turn, False)
    mixer = mixer_of(rt, hidden, layer)
    w = filled(mixer, 6, 1.2 / hidden ** 0.5)
    wd = doubles(w)
    g = torch.Generator().manual_seed(7)
    rows_of = {"a": torch.randn(350, hidden, generator=g).to(dtype), "b": torch.randn(60, hidden, generator=g).to(dtype)}
    plan = [{"a": na, "b": nb} for na, nb in [(0, 19), (13, 1), (150, 0), (1, 1), (1, 38), (2, 1), (1, 0), (22, 0), (160, 0)]]
    got = run_attention(rt, mixer, page, rows_of, plan, poison=True)
    for name, rows in rows_of.items():
        want, _ = plain.attention(rows.double(), wd, "p.", layer["mixer"], torch.arange(len(rows)), None)
        close(got[name], want.float(), dtype, f"request {name}", f32=5e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dv,page,chunk", [(16, 32, 8, 20), (64, 64, 16, 48), (64, 32, 16, 35), (24, 8, 4, 6), (128, 64, 16, 200), (64, 64, 16, 200)])
def test_one_key_at_the_chunk_edge(dtype, d, dv, page, chunk):
    """One key answers the last token's query far above all others and carries a value of its own.  The key is the
    first of the asking token's chunk, the last of the chunk before, at page borders and at the first tokens; the asking
    token is the first, the second and the last of its chunk and comes in a portion and alone.  An edge that is one token
    off changes the output by its whole size."""
    hidden, heads, kv = 48, 2, 1
    rt = Runtime(torch.device("cuda"), dtype)
    layer = attention(heads, kv, d, dv, 8.0 / d, chunk, rot(0, 10.0), False)
    mixer = mixer_of(rt, hidden, layer)
    w = filled(mixer, 8, 0.02)
    # queries and keys read channel 0 alone: a marked row (+1) meets a marked row with a score of 8 and an unmarked one
    # (-1) with -8; the values read channel 1
    for name in ("q", "k"):
        t = torch.zeros_like(w[name]); t[:, 0] = 1.0
        set_weight(mixer, w, name, t)
    t = torch.zeros_like(w["v"]); t[:, 1] = 2.0
    set_weight(mixer, w, "v", t)
    g = torch.Generator().manual_seed(1)
    set_weight(mixer, w, "o", torch.randn(w["o"].shape, generator=g) * 0.3)
    wd = doubles(w)
    checks, sizes = [], {True: [], False: []}
    start = 2 * chunk                                   # the asking token's chunk begins here
    for t in (start, start + 1, start + chunk - 1):
        for j in sorted({start, start - 1, max(t - 1, 0), start - chunk, start // page * page, start // page * page - 1, 0, t}):
            h = 0.01 * torch.randn(t + 1, hidden, generator=g)
            h[:, 0], h[:, 1] = -1.0, 1.0
            h[j, 0], h[j, 1] = 1.0, -5.0
            h[t, 0] = 1.0
            h = h.to(dtype)
            want = plain.attention(h.double(), wd, "p.", layer["mixer"], torch.arange(t + 1), None)[0].float()
            for tail in (0, 1, 5):                       # the asking token inside a portion, alone, after single tokens
                plan = [{"a": t + 1}] if tail == 0 else [{"a": t + 1 - tail}] + [{"a": 1}] * tail
                got = run_attention(rt, mixer, page, {"a": h}, plan, pages=-(-(t + 1) // page) + 1, poison=True)["a"]
                checks.append((f"key at {j}, asked at {t} (chunk from {start}), last {tail} tokens alone", got[-1:], want[-1:]))
            if j != t:
                sizes[j >= start].append(want[-1])
    size = max(float(x.abs().max()) for x in sizes[True] + sizes[False])
    assert min(float((a - b).abs().max()) for a in sizes[True] for b in sizes[False]) > 0.4 * size and size > 0.2
    for what, got, want in checks:
        err = float((got - want).abs().max())
        assert err <= (3e-5 if dtype == torch.float32 else 0.1) * size, f"{what}: differs by {err:.3g} (size {size:.3g})"


@pytest.mark.parametrize("dtype", DTYPES)
def test_values_blended_with_the_first_layers(dtype):
    """Three mixers in a row over one step's rows: the first leaves its values (its own number is not used), the second
    mixes nothing and leaves nothing behind, the third caches a blend with the first's; portions and single tokens of
    two requests, so that the kept rows are always those of the same step."""
    rt = Runtime(torch.device("cuda"), dtype)
    hidden, page = 48, 8
    layers = [attention(4, 2, 16, 32, 0.3, 9, rot(8, 100.0), True), attention(2, 2, 8, 32, 0.3, 11, None, False),
              attention(6, 2, 24, 32, 0.25, 20, rot(4, 50.0), True)]
    mixers, weights = [], []
    for i, layer in enumerate(layers):
        mixers.append(mixer_of(rt, hidden, layer, first=i == 0))
        weights.append(filled(mixers[-1], 30 + i, 0.17))
    set_weight(mixers[0], weights[0], "vmix", torch.tensor(5.0))
    set_weight(mixers[2], weights[2], "vmix", torch.tensor(0.375))
    g = torch.Generator().manual_seed(3)
    rows_of = [torch.randn(60, hidden, generator=g).to(dtype), torch.randn(41, hidden, generator=g).to(dtype)]
    want = []
    for rows in rows_of:
        pos, outs, first = torch.arange(len(rows)), [], None
        for i, (layer, w) in enumerate(zip(layers, weights)):
            out, v = plain.attention(rows.double(), doubles(w), "p.", layer["mixer"], pos, first if i == 2 else None)
            first = v if i == 0 else first
            outs.append(out.float())
        want.append(outs)
    cache = tw.CacheManager([(m.cache_need(), None) for m in mixers], page, 40, 2, 64, dtype, rt.device, prefix_cache=False, poison_freed=True)
    leases = [cache.admit(None), cache.admit(None)]
    at = {lease.slot: 0 for lease in leases}
    for counts in [(20, 5), (1, 7), (2, 1), (1, 1), (30, 0), (0, 27), (6, 0)]:
        live = [(r, n) for r, n in enumerate(counts) if n]
        for r, n in live:
            cache.ensure(leases[r], at[leases[r].slot] + n)
        cache.sync_tables()
        ctx = step_ctx(rt, [(leases[r].slot, n) for r, n in live], at)
        h = torch.cat([rows_of[r][at[leases[r].slot]:at[leases[r].slot] + n] for r, n in live]).cuda()
        for i, mixer in enumerate(mixers):
            out = dense_delta(ctx, mixer.forward(ctx, h, cache.view(i), True), dtype).float().cpu()
            cursor = 0
            for r, n in live:
                begin = at[leases[r].slot]
                close(out[cursor:cursor + n], want[r][i][begin:begin + n], dtype, f"mixer {i}, request {r} from {begin}", f32=5e-5)
                cursor += n
        assert int(ctx.status) == 0
        for r, n in live:
            at[leases[r].slot] += n
            cache.advance(leases[r], None, at[leases[r].slot])
    ctx = step_ctx(rt, [(leases[0].slot, 1)], {leases[0].slot: 0})
    with pytest.raises(RuntimeError, match="has left values"):      # nobody left values in this step
        mixers[2].forward(ctx, h[:1], cache.view(2), False)


KERNEL_CASES = [  # heads, kv heads, key size, value size, page, reach
    (8, 2, 128, 128, 16, -300), (4, 4, 64, 64, 16, -128), (6, 2, 128, 64, 32, -200), (8, 1, 64, 128, 16, -70), (4, 2, 64, 64, 64, 150),
    (28, 4, 128, 128, 16, 260), (2, 1, 128, 64, 256, -333), (4, 2, 64, 64, 16, 0), (5, 5, 128, 64, 8, -1000), (8, 2, 64, 32, 16, -200),
    (3, 1, 128, 32, 16, -90), (4, 4, 64, 32, 32, 0)]


@pytest.mark.parametrize("case", KERNEL_CASES)
@pytest.mark.parametrize("gated", [False, True])
def test_tensor_core_attention_against_the_exact_kernel(case, gated):
    """Every bfloat16 attention kernel -- mma.sync and tcgen05 prefill, split-KV decode through registers and by TMA with
    slices merged in one block, in a cluster and through scratch -- on the same paged cache as the exact kernel: chunks
    and windows that begin inside a page and inside a key tile, values of another size, gates.  Pages that the first row of
    a portion cannot see are not there at all, and what they would have held is NaN."""
    H, G, D, Dv, page, reach = case
    lengths, portions = [700, 333, 1000, 129, 641], [300, 333, 1, 1, 2]
    g = torch.Generator().manual_seed(D + Dv + page)
    blocks = [-(-n // page) for n in lengths]
    num_pages = sum(blocks) + 3
    order = torch.randperm(num_pages, generator=g)
    k = torch.randn(num_pages, G, page, D, generator=g).to(torch.bfloat16)
    v = torch.randn(num_pages, G, page, Dv, generator=g).to(torch.bfloat16)
    table = torch.full((len(lengths), max(blocks) + 1), -1, dtype=torch.int32)
    cursor, dead = 0, []
    for s, (n, b) in enumerate(zip(lengths, blocks)):
        pos = n - portions[s]
        first = max(0, pos - reach + 1) if reach > 0 else (pos - pos % -reach if reach < 0 else 0)
        for i in range(b):
            if i < first // page:
                dead.append(int(order[cursor + i]))
            else:
                table[s, i] = order[cursor + i]
        last = int(order[cursor + b - 1])                # behind the last token: whatever an earlier user left
        k[last, :, (n - 1) % page + 1:] = float("nan")
        v[last, :, (n - 1) % page + 1:] = float("nan")
        cursor += b
    dead += [int(p) for p in order[cursor:]]
    k[dead], v[dead] = float("nan"), float("nan")
    k, v, table = k.cuda(), v.cuda(), table.cuda()
    n_rows = sum(portions)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")     # noqa: E731
    starts = [sum(portions[:i]) for i in range(len(portions))]
    seq = [s for s, c in enumerate(portions) for _ in range(c)]
    positions = [lengths[s] - c + i for s, c in enumerate(portions) for i in range(c)]
    q = torch.randn(n_rows, H * D, generator=g).to(torch.bfloat16).cuda()
    gate = torch.rand(n_rows, H, generator=g).cuda() if gated else None
    slots = i32(list(range(len(lengths))))
    status, scale = i32([0]), 1.3 * D ** -0.5
    want = torch.full((n_rows, H * Dv), float("nan"), dtype=torch.bfloat16, device="cuda")
    ops.attention_generic(want, q, i32(positions), i32(seq), slots, table, k, v, n_rows, H, G, D, reach, scale, status, gate=gate)
    args = (i32(starts), i32(portions), i32(lengths), slots, table, k, v, len(lengths))
    single = [starts[2], starts[3]]
    several = [r for r in range(n_rows) if r not in single]

    def check(out, rows, what):
        assert int(status) == 0, what
        err = float((out[rows].float() - want[rows].float()).abs().max())
        assert err <= 2e-2 * float(want[rows].float().abs().max()), f"{what}: {err:.3g}"

    for name, kernel in (("mma.sync", ops.attention_prefill), ("tcgen05", ops.attention_prefill_tcgen05)):
        out = torch.full_like(want, float("nan"))
        kernel(out, q, *args, max(portions), H, G, D, reach, scale, True, status, gate=gate)
        check(out, several, name)
        assert bool(torch.isnan(out[single].float()).all())
    for nsplit, scratch_merge in ((1, False), (3, False), (3, True), (20, False)):
        scratch = torch.full((ops.decode_scratch_floats(H, Dv),), float("nan"), device="cuda")
        counters = torch.zeros(ops.decode_counter_ints(len(lengths), G, H // G), dtype=torch.int32, device="cuda")
        out = torch.full_like(want, float("nan"))
        ops.attention_decode(out, q, *args, H, G, D, reach, scale, nsplit, scratch, counters, status, merge_in_scratch=scratch_merge, gate=gate)
        check(out, single, f"decode, {nsplit} slices")
        if ops.decode_tma_supported(torch.bfloat16, D, page, Dv):
            out = torch.full_like(want, float("nan"))
            ops.attention_decode_tma(out, q, None, None, None, False, *args, H, G, D, reach, scale, nsplit, scratch, counters, status,
                                     merge_in_scratch=scratch_merge, gate=gate)
            check(out, single, f"TMA decode, {nsplit} slices")
            assert bool(torch.isnan(out[several].float()).all())


# ---------------------------------------------------------------------------
# feed-forwards alone
# ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff", [(64, 40), (36, 27), (128, 200), (40, 9), (512, 1024)])
@pytest.mark.parametrize("forced", [None, "stream", "pair"])
def test_gelu_feed_forward_with_biases_alone(dtype, hidden, ff, forced, monkeypatch):
    """Few rows (the weight-streaming kernel), some (the persistent tcgen05 kernel where it is forced, else the
    library), many (block pairs where forced): the biases stand with the right rows of the packed matrix, and gelu has
    the tanh form (at arguments where the exact form differs by more than the bound in 32 bits)."""
    if forced == "stream":
        monkeypatch.setenv("TESSWEAVE_STREAM_MIN_WEIGHTS", "1")
    elif forced == "pair":
        monkeypatch.setenv("TESSWEAVE_PAIR_GEMM", "force")
    rt = Runtime(torch.device("cuda"), dtype)
    typed, layer = typed_layer(hidden, attention(1, 1, 8, 8, 0.3, 4, None, False, dense(ff)))
    part = build_part("feed_forward", feed_forward_spec(typed, layer.mlp), rt)
    w = filled(part, 5, 1.0 / hidden ** 0.5)
    for name in ("gate.b", "up.b", "down.b"):
        set_weight(part, w, name, torch.randn(w[name].shape, generator=torch.Generator().manual_seed(len(name))))
    wd = doubles(w)
    h = torch.randn(300, hidden, generator=torch.Generator().manual_seed(2)).to(dtype)
    for n in (1, 7, 8, 9, 33, 64, 300):
        ctx = ctx_of(rt, list(range(n)), [0] * n, [0], [0], [n], [n])
        got = dense_delta(ctx, part.forward(ctx, h[:n].cuda()), dtype).float().cpu()
        assert int(ctx.status) == 0
        close(got, plain.dense(h[:n].double(), wd, "p.").float(), dtype, f"{n} rows", f32=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff", [(64, 40), (36, 27), (128, 200), (40, 9), (512, 1024)])
@pytest.mark.parametrize("forced", [None, "stream", "pair"])
@pytest.mark.parametrize("function", ["relu_squared", "gelu_tanh", "silu"])
def test_feed_forward_of_two_matrices_alone(dtype, hidden, ff, forced, function, monkeypatch):
    if forced == "stream":
        monkeypatch.setenv("TESSWEAVE_STREAM_MIN_WEIGHTS", "1")
    elif forced == "pair":
        monkeypatch.setenv("TESSWEAVE_PAIR_GEMM", "force")
    rt = Runtime(torch.device("cuda"), dtype)
    part = build_part("feed_forward", PartSpec("plain_mlp", {"hidden": hidden, "intermediate": ff, "activation": function}), rt)
    w = fill(part, 5, 1.5 / hidden ** 0.5)
    f = {"relu_squared": plain.relu_squared, "gelu_tanh": plain.gelu_tanh, "silu": lambda z: z * torch.sigmoid(z)}[function]
    h = torch.randn(300, hidden, generator=torch.Generator().manual_seed(2)).to(dtype)
    for n in (1, 8, 9, 64, 300):
        ctx = ctx_of(rt, list(range(n)), [0] * n, [0], [0], [n], [n])
        got = dense_delta(ctx, part.forward(ctx, h[:n].cuda()), dtype).float().cpu()
        assert int(ctx.status) == 0
        want = f(h[:n].double() @ w["up"].double().T) @ w["down"].double().T
        close(got, want.float(), dtype, f"{n} rows", f32=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,experts,top,ff,shared", [(64, 6, 2, 40, 24), (40, 3, 1, 20, None), (36, 5, 5, 9, 7), (128, 10, 4, 88, 136),
                                                          (48, 1, 1, 16, 16), (64, 40, 3, 24, 64)])
def test_experts_without_gates_alone(dtype, hidden, experts, top, ff, shared):
    """Scores over all experts, the largest kept without renormalising, the square of relu, the shared expert times its
    sigmoid; sorted by expert (bfloat16, several rows) and pair by pair; rows whose choice no rounding can turn."""
    rt = Runtime(torch.device("cuda"), dtype)
    mlp = moe(experts, top, ff, shared)
    typed, layer = typed_layer(hidden, attention(1, 1, 8, 8, 0.3, 4, None, False, mlp))
    part = build_part("feed_forward", feed_forward_spec(typed, layer.mlp), rt)
    w = filled(part, 14, 1.2 / hidden ** 0.5)
    wd = doubles(w)
    rows = 37
    h = torch.randn(rows, hidden, generator=torch.Generator().manual_seed(2)).to(dtype)
    want = plain.mixture(h.double(), wd, "p.", mlp).float()
    chosen_want, weight_want = plain.route(h.double(), wd, "p.", top)
    ctx = ctx_of(rt, list(range(rows)), [0] * rows, [0], [0], [rows], [rows])
    chosen, weight, _ = part.route(ctx, h.cuda())
    scores = torch.softmax(h.double() @ wd["p.router"].T, -1)
    sure = torch.ones(rows, dtype=torch.bool)
    if top < experts:
        ranked = scores.sort(dim=-1, descending=True).values
        sure = (ranked[:, top - 1] - ranked[:, top]) > 2e-3
        assert float(weight_want.sum(-1).max()) < 0.99             # what is left out is felt
    assert int(sure.sum()) >= rows // 2
    assert torch.equal(chosen.cpu().long().sort(-1).values[sure], chosen_want.sort(-1).values[sure])
    close(weight.cpu()[sure], torch.gather(scores, 1, chosen.cpu().long())[sure].float(), torch.float32, "weights of the chosen",
          f32=1e-2 if dtype == torch.bfloat16 else 1e-5)
    for n in (rows, 2, 1):
        one = ctx_of(rt, list(range(n)), [0] * n, [0], [0], [n], [n])
        got = dense_delta(one, part.forward(one, h[:n].cuda()), dtype).float().cpu()
        close(got[sure[:n]], want[:n][sure[:n]], dtype, f"experts, {n} rows")


# ---------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------
def settle_router(folder):
    """For bfloat16 runs: a router whose choice no rounding can turn.  Channel 0 of every embedding row becomes one
    number that stays the largest part of it, and the router's column of that channel sets the experts apart in an order
    of the layer's own by more than a token's other channels (whose columns are shrunk) move them.  (The choice per
    token is what the float32 runs, whose routers are random, and the test of the part alone check.)"""
    from safetensors.torch import load_file, save_file
    t = load_file(str(folder / "model.safetensors"))
    t["embed"][:, 0] = 4.0
    for name in sorted(t):
        if name.endswith(".mlp.router"):
            g = torch.Generator().manual_seed(len(name) + t[name].shape[0])
            t[name] = (0.05 * t[name].float()).to(t[name].dtype)
            t[name][:, 0] = (torch.randperm(t[name].shape[0], generator=g).float() * 0.2).to(t[name].dtype)
    save_file(t, str(folder / "model.safetensors"), metadata={"format": "pt"})
    return folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """(name, dtype) -> model folder; the bfloat16 runs get a copy whose routers are settled."""
    tmp = tmp_path_factory.mktemp("varivik")
    out = {}
    for name, cfg in VARIVIK_CONFIGS.items():
        for dtype in ("float32", "bfloat16"):
            folder = tw.write_random_model(tmp / f"{name}_{dtype}", cfg, seed=VARIVIK_SEEDS[name], std=VARIVIK_STD[name])
            out[name, dtype] = settle_router(folder) if dtype == "bfloat16" else folder
    return out


LENGTHS = [70, 1, 45, 100, 2, 33, 64, 129]


def requests_for(name):
    return {f"r{i}": random_tokens(VARIVIK_CONFIGS[name]["vocab"], n, 20 + i) for i, n in enumerate(LENGTHS)}


@pytest.fixture(scope="module")
def plain_rows(folders):
    return {key: {rid: plain.logits_of(folder, t).numpy() for rid, t in requests_for(key[0]).items()}
            for key, folder in folders.items()}


def compare(rows, want, dtype, what):
    """Every logits row against the plain one (float64), by the root mean square over the vocabulary (mean taken off)
    against the row's spread: 5e-5 in float32; in bfloat16 3 % for the median row and 10 % for every row.  A key outside
    its chunk, a wrong page or values that are not blended move rows by a large part of their size."""
    errors = []
    for (rid, p), row in rows.items():
        assert np.isfinite(row).all(), f"{what}: {rid}[{p}] is not finite"
        errors.append((row_error(row, want[rid][p]), rid, p))
    worst = max(errors)
    median = float(np.median([e for e, _, _ in errors]))
    if dtype == "float32":
        assert worst[0] <= 5e-5, f"{what}: {worst[1]}[{worst[2]}] differs by {worst[0]:.3g} of the row's spread"
    else:
        assert median <= 3e-2, f"{what}: the median row differs by {median:.3g}"
        assert worst[0] <= 1e-1, f"{what}: {worst[1]}[{worst[2]}] differs by {worst[0]:.3g} of the row's spread"


SCHEDULES = {
    "whole": schedule_whole,
    "tail": schedule_tail,
    "portions": schedule_portions,
    "one_by_one": lambda r: schedule_portions({k: v for k, v in r.items() if len(v) <= 70}, sizes=(1,)),
    "mixed": lambda r: schedule_mixed(r, live=4, seed=1),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_every_cutting_gives_the_plain_logits(name, dtype, folders, plain_rows, tmp_path):
    """Whole prompts; most of a prompt and its last 32 tokens one by one; portions down to two tokens; token by
    token from the first; four live requests in mixed batches with so few pages and slots that both are used
    again (freed pages are filled with NaN first)."""
    reqs = requests_for(name)
    for kind, make in SCHEDULES.items():
        steps = make(reqs)
        rows = replay_in_process(folders[name, dtype], dtype, steps, tmp_path / kind, block_size=VARIVIK_PAGE[name],
                                 max_tokens=max_live_tokens(steps))
        assert rows, kind
        compare(rows, plain_rows[name, dtype], dtype, f"{name} {kind}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_and_cuts_do_not_change_a_request(dtype, folders, tmp_path):
    """A request's logits in a mixed batch, or cut into portions, equal those it gets alone, to rounding."""
    reqs = requests_for("A")
    folder = folders["A", dtype]
    alone = replay_in_process(folder, dtype, schedule_whole(reqs), tmp_path / "alone", block_size=8)
    for kind, steps in (("mixed", schedule_mixed(reqs, live=4, seed=3)), ("portions", schedule_portions(reqs))):
        got = replay_in_process(folder, dtype, steps, tmp_path / kind, block_size=8)
        worst = max(row_error(row, alone[key]) for key, row in got.items())
        assert worst <= (5e-5 if dtype == "float32" else 0.1), (kind, worst)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_used_again(dtype, folders):
    """One request slot and barely enough pages: each request gets the slot and the pages its predecessor gave back,
    with the predecessor's keys and values still in them."""
    from tessweave_engine_b200.engine.runner import ModelRunner, StepEntry
    name = "A"
    model = tw.load_model(folders[name, dtype], dtype, "cuda")
    cache = tw.CacheManager(model.cache_needs(), VARIVIK_PAGE[name], 9, 1, 72, model.runtime.dtype, model.runtime.device,
                            prefix_cache=False)
    runner = ModelRunner(model, cache, 72, 1, cuda_graphs=False)
    config, weights = plain.read_folder(folders[name, dtype], torch.float64)
    for i, n in enumerate([70, 64, 3, 71]):
        tokens = random_tokens(config["vocab"], n, 40 + i)
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
        want = plain.forward(config, weights, tokens).numpy()
        compare({("r", cut + k): got[k] for k in range(n - cut)}, {"r": want}, dtype, f"request {i} in a used slot")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_past_chunks_and_pages(dtype, folders, tmp_path):
    """A short prompt and 300 tokens one by one: chunks begin and end among decoded tokens only, and the pages of
    finished chunks are given back and used again on the way."""
    name = "C"
    toks = random_tokens(VARIVIK_CONFIGS[name]["vocab"], 310, 77)
    steps = schedule_tail({"long": toks}, tail=300)
    rows = replay_in_process(folders[name, dtype], dtype, steps, tmp_path / "out", block_size=VARIVIK_PAGE[name], max_tokens=384)
    compare(rows, {"long": plain.logits_of(folders[name, dtype], toks).numpy()}, dtype, "long decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_of_hundreds_of_tokens_past_chunks(dtype, tmp_path):
    """Head sizes of the kernels fed by TMA, chunks of 70 and 150 and none, prompts of 420 and 190 tokens: whole, with
    the last 40 tokens one by one, and in mixed batches with portions of more than a hundred tokens."""
    cfg = VARIVIK_E
    folder = tw.write_random_model(tmp_path / "model", cfg, seed=31, std=0.1)
    if dtype == "bfloat16":
        settle_router(folder)
    reqs = {"long": random_tokens(cfg["vocab"], 420, 5), "mid": random_tokens(cfg["vocab"], 190, 6), "short": random_tokens(cfg["vocab"], 37, 7)}
    want = {rid: plain.logits_of(folder, t).numpy() for rid, t in reqs.items()}
    for kind, steps in (("whole", schedule_whole(reqs)), ("tail", schedule_tail(reqs, tail=40)),
                        ("mixed", schedule_mixed(reqs, live=3, seed=2, prefill=(33, 2, 150, 5, 128, 16)))):
        rows = replay_in_process(folder, dtype, steps, tmp_path / kind, block_size=16, max_tokens=max_live_tokens(steps))
        compare(rows, want, dtype, f"E {kind}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_engine(name, dtype, folders):
    """``generate`` (scheduler, continuous batching, CUDA graphs, look-ahead) against the plain greedy loop;
    every chosen token must be the plain implementation's best on that path, or nearly."""
    prompts = [random_tokens(VARIVIK_CONFIGS[name]["vocab"], n, 60 + n) for n in (21, 5, 40)]
    model = tw.load_model(folders[name, dtype], dtype, "cuda")
    out = tw.generate(model, prompts, max_tokens=30, ignore_eos=True,
                      engine_config=tw.EngineConfig(block_size=VARIVIK_PAGE[name], kv_blocks=40, max_context=128, max_active=2,
                                                    prefill_chunk=16))
    config, weights = plain.read_folder(folders[name, dtype], torch.float64)
    for p, o in zip(prompts, out):
        assert len(o) == 30
        logits = plain.forward(config, weights, p + o).float()
        for i, t in enumerate(o):
            row = logits[len(p) + i - 1]
            gap = float(row.max() - row[t])
            spread = float(row.std())
            assert gap <= (1e-4 if dtype == "float32" else 0.2) * spread, f"token {i} lies {gap:.3g} below the best (spread {spread:.3g})"

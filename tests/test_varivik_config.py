"""The Varivik configuration gate and spec builder (no GPU): what is read from where, what is refused; the cache manager
with chunks; and the plain implementation against itself where a mechanism can be written two ways."""
import copy
import json
import math
import random

import pytest
import torch

import plain_varivik as plain
import tessweave_engine_b200 as tw
from tessweave_engine_b200.cache import CacheManager
from tessweave_engine_b200.config import ConfigError, resolve
from tessweave_engine_b200.models import Model
from tessweave_engine_b200.parts import PagedKV, Runtime
from tessweave_engine_b200.parts.positions import banded_frequencies
from tiny_varivik import VARIVIK_CONFIGS, VARIVIK_E, bands

ALL = {**VARIVIK_CONFIGS, "E": VARIVIK_E}


def meta_model(cfg):
    typed, spec = resolve(cfg)
    return typed, spec, Model(spec, Runtime(torch.device("meta"), torch.float32), config=typed)


@pytest.mark.parametrize("name", list(ALL))
def test_tensor_names_and_shapes(name):
    cfg = ALL[name]
    typed, spec, model = meta_model(cfg)
    assert len(spec.layers) == len(spec.schedule) == len(cfg["layers"])
    decls = model.weight_decls()
    width = cfg["width"]
    want = {"embed": (cfg["vocab"], width), "final.norm": (width,)}
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        want[p + "norm1"] = (width,)
        want.update({p + "mix.q": (H * D, width), p + "mix.k": (G * D, width), p + "mix.v": (G * Dv, width), p + "mix.g": (H, width),
                     p + "mix.o": (width, H * Dv)})
        if m["v_mix"]:
            want[p + "mix.vmix"] = ()
        if mlp is None:
            continue
        want[p + "norm2"] = (width,)
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            want.update({p + "mlp.gate": (F, width), p + "mlp.gate.b": (F,), p + "mlp.up": (F, width), p + "mlp.up.b": (F,),
                         p + "mlp.down": (width, F), p + "mlp.down.b": (width,)})
        else:
            want[p + "mlp.router"] = (mlp["router"]["experts"], width)
            for e in range(mlp["router"]["experts"]):
                want.update({f"{p}mlp.e{e}.up": (mlp["expert"]["ff"], width), f"{p}mlp.e{e}.down": (width, mlp["expert"]["ff"])})
            if "shared" in mlp:
                F = mlp["shared"]["ff"]
                want.update({p + "mlp.shared.up": (F, width), p + "mlp.shared.down": (width, F), p + "mlp.shared.sg": (1, width)})
    assert {k: tuple(d.shape) for k, d in decls.items()} == want


def test_constants_reach_the_parts():
    _, spec, model = meta_model(VARIVIK_CONFIGS["A"])
    mix = [b.mixer for b in model.blocks]
    assert [m.chunk for m in mix] == [9, 20, None, 33, 7] and all(m.window is None for m in mix)
    assert [m.reach for m in mix] == [-9, -20, 0, -33, -7]
    assert [m.scale for m in mix] == [0.3, 0.2, 0.35, 0.25, 0.17]
    assert [m.value_mix and m.value_mix["role"] for m in mix] == [None, "first", "mix", "mix", "mix"]
    assert mix[0].position.bands == {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64.0} and mix[1].position.bands is None
    assert [m.position.kind for m in mix] == ["rope_interleaved"] * 3 + ["none", "rope_interleaved"]
    assert mix[0].position.rotary_plan(16).rot_dims == 8 and mix[1].position.theta == 5e4
    ff = [b.feed_forward for b in model.blocks]
    assert ff[3] is None and (ff[0].intermediate, ff[4].intermediate) == (40, 24)
    assert (ff[1].experts, ff[1].top, ff[1].intermediate, ff[1].shared.intermediate) == (6, 2, 24, 40) and ff[2].shared is None
    assert ff[1].score_all and ff[1].weight_scale == 1.0 and ff[1].correction is None and not ff[1].gated
    assert model.head.tied and model.final_norm.eps == 1e-5
    _, _, d = meta_model(VARIVIK_CONFIGS["D"])
    assert [b.mixer.value_mix and b.mixer.value_mix["role"] for b in d.blocks] == [None, None, "first"]


def test_cache_needs():
    """Keys and values of their own sizes, and the chunk goes to the cache manager; layers of one need share pages."""
    _, _, model = meta_model(VARIVIK_CONFIGS["A"])
    needs = [n for n, _ in model.cache_needs()]
    assert needs[0] == PagedKV(2, 16, None, 32, chunk=9) and needs[3] == PagedKV(2, 16, None, None, chunk=33)
    assert needs[2] == PagedKV(2, 8, None, 16)
    assert model.cache_bytes_per_token(2) == 2 * 2 * (16 + 32 + 24 + 16 + 8 + 16 + 16 + 16 + 32 + 16)
    assert model.state_bytes_per_request() == 0


def edit(cfg, path, value):
    cfg = copy.deepcopy(cfg)
    node = cfg
    for key in path[:-1]:
        node = node[key]
    if value is KeyError:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "mamba", "not implemented"),
    (("layers", 0, "mixer", "rot", "dims"), 5, "even"),
    (("layers", 0, "mixer", "rot", "dims"), 18, "head size"),
    (("layers", 0, "mixer", "rot", "base"), 0.0, "positive"),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0, "positive"),
    (("layers", 0, "mixer", "rot", "scaling", "high"), 1.0, "above low"),
    (("layers", 0, "mixer", "mask", "size"), 0, "positive"),
    (("layers", 0, "mixer", "v_mix"), "yes", "true or false"),
    (("layers", 0, "mixer", "v_mix"), True, "equal in all"),
    (("layers", 0, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 0, "mixer", "vdim"), 1300, "not supported"),
    (("layers", 0, "mixer", "heads"), KeyError, "heads"),
    (("layers", 0, "mlp", "kind"), "sparse", "not implemented"),
    (("layers", 0, "mlp", "ff"), 0, "positive"),
    (("layers", 1, "mlp", "router", "top"), 7, "top exceeds"),
    (("layers", 1, "mlp", "shared", "ff"), -1, "positive"),
    (("norm", "eps"), 0.0, "positive"),
    (("width",), 0, "positive"),
    (("layers",), [], "non-empty"),
])
def test_what_the_gate_refuses(path, value, word):
    with pytest.raises(ConfigError) as e:
        resolve(edit(VARIVIK_CONFIGS["A"], path, value))
    assert word in str(e.value)


def test_written_weights_are_read_back(tmp_path):
    """A folder written from a configuration holds every tensor the model declares (a number without axes among them),
    and the plain reader sees them."""
    cfg = VARIVIK_CONFIGS["D"]
    folder = tw.write_random_model(tmp_path / "m", cfg, seed=3, std=0.2)
    stored, w = plain.read_folder(folder, torch.float64)
    _, _, model = meta_model(cfg)
    assert set(w) == set(model.weight_decls()) and w["l2.mix.vmix"].shape == ()
    logits = plain.forward(stored, w, [1, 5, 2, 40, 7])
    assert logits.shape == (5, 53) and bool(torch.isfinite(logits).all())


@pytest.mark.parametrize("dims,base,scaling", [(32, 5e4, bands(4.0, 1.0, 4.0, 64)), (16, 100.0, bands(2.0, 0.5, 2.0, 16)),
                                               (8, 10.0, bands(3.0, 0.0, 1.0, 9)), (64, 1e6, bands(8.0, 1.0, 4.0, 8192))])
def test_banded_rates(dims, base, scaling):
    """By turns over the original length (the engine's form) and by wavelengths (the plain form) the rates are the
    same; the fast pairs keep their rate, the slow ones lose the factor, and the bands meet without a jump."""
    got = banded_frequencies(base, dims, scaling)
    want = plain.turning_rates(dims, base, scaling)
    free = plain.turning_rates(dims, base, None)
    assert max(abs(a - b) / b for a, b in zip(got, want)) < 1e-12
    kinds = set()
    for f, g in zip(free, got):
        turns = scaling["original"] * f / (2 * math.pi)
        kind = "kept" if turns >= scaling["high"] else "slowed" if turns <= scaling["low"] else "between"
        kinds.add(kind)
        if kind != "between":
            assert abs(g - (f if kind == "kept" else f / scaling["factor"])) < 1e-12 * f
        else:
            assert f / scaling["factor"] < g < f
    if scaling["low"] > 0:
        assert "kept" in kinds or "between" in kinds
        assert "slowed" in kinds


def test_plain_chunks_and_mixed_values():
    seen = plain.visible(7, 3)
    assert seen.tolist() == [[i >= j and i // 3 == j // 3 for j in range(7)] for i in range(7)]
    assert bool(plain.visible(5, None).equal(torch.ones(5, 5).tril().bool()))
    assert plain.visible(4, 1).equal(torch.eye(4).bool())
    v, first = torch.tensor([2.0]), torch.tensor([10.0])
    assert float(plain.mix_values(v, first, 0.25)) == 4.0


# ---------------------------------------------------------------------------
# the cache manager with chunks
# ---------------------------------------------------------------------------
def test_first_needed_key():
    need = PagedKV(1, 8, chunk=5)
    assert [need.first_needed(p) for p in range(11)] == [0] * 5 + [5] * 5 + [10] and need.span == 5
    assert [PagedKV(1, 8, window=3).first_needed(p) for p in range(5)] == [0, 0, 0, 1, 2]
    assert PagedKV(1, 8).first_needed(100) == 0 and PagedKV(1, 8).span is None


@pytest.mark.parametrize("chunk,page", [(10, 4), (8, 4), (3, 4), (1, 4), (16, 8), (7, 2)])
def test_pages_of_a_finished_chunk_are_given_back(chunk, page):
    """After every step a request holds exactly the pages from the first key that its next token sees on; the promise
    made at admission covers them for every way of cutting; other requests get what it gave back."""
    rng = random.Random(chunk * 100 + page)
    step_most = 6
    m = CacheManager([(PagedKV(1, 8, chunk=chunk), None)], page, 64, 3, 200, torch.float32, "cpu", prefix_cache=True)
    assert not m.prefix_cache                       # a chunk's pages are gone later: nothing to share by hash
    most = m.pages_needed(100, step_most)[0]
    assert most <= -(-(chunk + step_most) // page) + 1
    leases = [m.admit(None, reserve_tokens=100, step_tokens=step_most) for _ in range(3)]
    at = [0, 0, 0]
    while min(at) < 100:
        i = rng.choice([k for k in range(3) if at[k] < 100])
        n = min(rng.randint(1, step_most), 100 - at[i])
        m.ensure(leases[i], at[i] + n)
        m.check_writable(leases[i].slot, at[i], at[i] + n)
        first = at[i] - at[i] % chunk
        table = leases[i].tables[0]
        assert all(table[b] >= 0 for b in range(first // page, -(-(at[i] + n) // page))), "a page the step reads is missing"
        at[i] += n
        m.advance(leases[i], None, at[i])
        m.check_invariants()
        first = at[i] - at[i] % chunk
        held = [b for b, p in enumerate(leases[i].tables[0]) if p >= 0]
        assert all(b >= first // page for b in held) and len(held) <= most
    for lease in leases:
        m.release(lease)
    assert len(m.groups[0].free) == 64 and m.groups[0].promised == 0

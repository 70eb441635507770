"""The Bavetar configuration gate and spec builder (no GPU): what is read from where, what is refused; and the plain
implementation against itself where a mechanism can be written two ways."""
import copy
import json

import pytest
import torch

import plain_bavetar as plain
import tessweave_engine_b200 as tw
from tessweave_engine_b200.config import ConfigError, resolve
from tessweave_engine_b200.models import Model
from tessweave_engine_b200.parts import FixedState, PagedKV, Runtime
from tiny_bavetar import BAVETAR_A, BAVETAR_CONFIGS, BAVETAR_E, mamba, moe


def meta_model(cfg):
    typed, spec = resolve(cfg)
    return typed, spec, Model(spec, Runtime(torch.device("meta"), torch.float32), config=typed)


@pytest.mark.parametrize("name", list(BAVETAR_CONFIGS) + ["E"])
def test_tensor_names_and_shapes(name):
    cfg = {**BAVETAR_CONFIGS, "E": BAVETAR_E}[name]
    typed, spec, model = meta_model(cfg)
    assert len(spec.layers) == len(spec.schedule) == len(cfg["layers"])
    decls = model.weight_decls()
    names = set(decls)
    width = cfg["width"]
    assert {"embed", "final.norm"} <= names and not any(n.startswith("head") for n in names)     # the head is the embedding
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}", layer["mixer"], layer["mlp"]
        assert f"{p}.norm1" in names and (f"{p}.norm2" in names) == (mlp is not None)
        mine = {n[len(p) + 5:]: decls[n].shape for n in names if n.startswith(f"{p}.mix.")}
        H, Dv = m["heads"], m["vdim"]
        if layer["type"] == "latent_attention":
            D, R, Q, C = m["dim"], m["rot_dim"], m["q_rank"], m["kv_rank"]
            assert mine == {"dq": (Q, width), "dq.norm": (Q,), "uq": (H * (D + R), Q), "dkv": (C + R, width), "dkv.norm": (C,),
                            "uk": (H * D, C), "uv": (H * Dv, C), "g": (H, width), "sink": (H,), "o": (width, H * Dv)}
        else:
            N, G, taps = m["state"], m["groups"], m["conv"]
            channels = H * Dv + 2 * G * N
            assert mine == {"in": (H * Dv + channels + H, width), "conv": (channels, taps), "conv.b": (channels,), "dt_bias": (H,),
                            "A_log": (H,), "D": (H,), "norm": (H * Dv,), "o": (width, H * Dv)}
        ff = {n[len(p) + 5:]: decls[n].shape for n in names if n.startswith(f"{p}.mlp.")}
        if mlp is None:
            assert not ff
        elif mlp["kind"] == "dense":
            assert ff == {"up": (mlp["ff"], width), "down": (width, mlp["ff"])}
        else:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            want = {"router": (E, width)}
            for e in range(E):
                want.update({f"e{e}.gate": (F, width), f"e{e}.up": (F, width), f"e{e}.down": (width, F)})
            assert ff == want


def test_cache_needs():
    """A latent layer keeps one row of kv_rank + rot_dim values per token that serves as key and value; a recurrent layer
    a matrix per head and the convolution's last inputs."""
    _, spec, model = meta_model(BAVETAR_A)
    needs = [n for n, _ in model.cache_needs()]
    assert needs[0] == FixedState(4 * 16 * 16 + (4 * 16 + 2 * 2 * 16) * 3)
    assert needs[1] == PagedKV(1, 48, None, None, values_are_keys=True)
    assert needs[4] == FixedState(3 * 8 * 8 + (3 * 8 + 2 * 3 * 8) * 1)
    assert model.cache_bytes_per_token(2) == 2 * (48 + 32 + 32)
    assert model.state_bytes_per_request() == 4 * sum(n.numel for n in needs if isinstance(n, FixedState))
    _, _, b = meta_model(BAVETAR_CONFIGS["B"])
    assert [n.numel for n, _ in b.cache_needs() if isinstance(n, FixedState)] == [3 * 10 * 6 + (18 + 60) * 5, 4 * 7 * 5]     # one tap: nothing kept


def test_constants_reach_the_parts():
    typed, spec, model = meta_model(BAVETAR_A)
    assert model.head.softcap == 12.0 and model.head.scale == 1.5 and spec.tie_word_embeddings
    rec, lat = model.blocks[0].mixer, model.blocks[1].mixer
    assert (rec.n_groups, rec.taps, rec.norm_groups, rec.key_dim, rec.eps) == (2, 4, 1, 16, 1e-5)
    assert (lat.scale, lat.kv_rank, lat.rot_dim, lat.eps, lat.window, lat.gate) == (0.2, 40, 8, 1e-5, None, "heads")
    assert lat.sink is not None and lat.position.yarn is None
    ff = model.blocks[0].feed_forward
    assert (ff.experts, ff.top, ff.weight_scale, ff.groups, ff.renormalise, ff.score_all, ff.identity) == (8, 3, 2.0, (4, 2), True, True, 0)
    assert model.blocks[0].norm2 is not None and model.blocks[4].norm2 is None
    assert "l4.norm2" in model.redundant_names() and "l0.norm2" not in model.redundant_names()
    _, _, b = meta_model(BAVETAR_CONFIGS["B"])
    assert b.head.softcap is None and b.head.scale == 1.0 and b.blocks[0].feed_forward.groups is None


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
    (("layers", 0, "type"), "gla", "not implemented"),
    (("layers", 0, "mixer", "groups"), 3, "multiple"),
    (("layers", 0, "mixer", "norm_groups"), 7, "divide"),
    (("layers", 0, "mixer", "state"), 300, "does not fit"),
    (("layers", 0, "mixer", "vdim"), 256, "does not fit"),
    (("layers", 0, "mixer", "conv"), 18, "taps"),
    (("layers", 0, "mixer", "heads"), KeyError, "heads"),
    (("layers", 0, "mlp", "kind"), "conv", "not implemented"),
    (("layers", 0, "mlp", "router", "top"), 9, "top exceeds"),
    (("layers", 0, "mlp", "router", "groups", "count"), 3, "not possible"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 1, "not possible"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 5, "not possible"),
    (("layers", 1, "mixer", "rot", "dims"), 4, "rot_dim"),
    (("layers", 1, "mixer", "rot_dim"), 7, "even"),
    (("layers", 1, "mixer", "kv_rank"), 1020, "not supported"),
    (("layers", 1, "mixer", "rot", "base"), 0.0, "positive"),
    (("layers", 1, "mixer", "mask"), {"size": 4}, "every earlier token"),
    (("layers", 1, "mixer", "rot", "scaling"), {"factor": 2.0}, "scaling"),
    (("layers", 1, "mlp", "ff"), 0, "positive"),
    (("norm", "eps"), 0.0, "positive"),
    (("logit_softcap",), -2.0, "positive"),
    (("logit_scale",), "two", "finite"),
    (("width",), 0, "positive"),
    (("layers",), [], "non-empty"),
])
def test_what_the_gate_refuses(path, value, word):
    with pytest.raises(ConfigError) as e:
        resolve(edit(BAVETAR_A, path, value))
    assert word in str(e.value)


def test_written_weights_are_read_back(tmp_path):
    """A folder written from a configuration holds every tensor the model declares, and the plain reader sees them."""
    cfg = BAVETAR_CONFIGS["D"]
    folder = tw.write_random_model(tmp_path / "m", cfg, seed=3, std=0.2)
    _, w = plain.read_folder(folder, torch.float64)
    _, _, model = meta_model(cfg)
    assert set(w) == set(model.weight_decls())
    logits = plain.forward(json.loads((folder / "config.json").read_text()), w, [1, 5, 2, 40, 7])
    assert logits.shape == (5, 53) and bool(torch.isfinite(logits).all()) and float(logits.abs().max()) < 5.0    # the cap


# ---------------------------------------------------------------------------
# the plain implementation
# ---------------------------------------------------------------------------
def test_plain_recurrence_as_one_sum():
    """Unrolled, y_t = sum over s <= t of exp(-rate (dt_{s+1} + ... + dt_t)) dt_s (c_t . b_s) x_s + skip x_t."""
    g = torch.Generator().manual_seed(2)
    T, H, N, Dv = 19, 3, 5, 4
    x, b, c = (torch.randn(T, H, d, generator=g, dtype=torch.float64) for d in (Dv, N, N))
    dt = torch.rand(T, H, generator=g, dtype=torch.float64)
    rate, skip = torch.rand(H, generator=g, dtype=torch.float64) + 0.2, torch.randn(H, generator=g, dtype=torch.float64)
    total = torch.cumsum(dt, 0)
    decay = torch.exp(-rate * (total[:, None] - total[None, :]))                      # [t, s, H]
    decay = decay * (torch.arange(T)[None, :] <= torch.arange(T)[:, None])[:, :, None]
    want = torch.einsum("tsh,sh,thn,shn,shv->thv", decay, dt, c, b, x) + skip[:, None] * x
    got = plain.state_space_recurrence(x, b, c, dt, rate, skip)
    assert float((got - want).abs().max()) < 1e-12


def test_plain_convolution_by_hand():
    x = torch.arange(1.0, 7.0, dtype=torch.float64).view(3, 2)           # rows (1, 2), (3, 4), (5, 6)
    weight = torch.tensor([[10.0, 1.0], [0.5, -1.0]], dtype=torch.float64)
    bias = torch.tensor([0.25, 0.0], dtype=torch.float64)
    pre = torch.tensor([[1.25, -2.0], [13.25, -3.0], [35.25, -4.0]], dtype=torch.float64)
    assert torch.allclose(plain.causal_convolution(x, weight, bias), pre * torch.sigmoid(pre))


def test_plain_softmax_with_sinks():
    s = torch.tensor([[[0.0, 9.0], [1.0, 2.0]], [[3.0, 9.0], [0.0, 0.0]]], dtype=torch.float64)
    sink = torch.tensor([0.5, -1.0], dtype=torch.float64)
    p = plain.softmax_with_sink(s, sink)
    for head in range(2):
        e = torch.exp(s[head])
        assert torch.allclose(p[head, 0], torch.stack([e[0, 0] / (e[0, 0] + torch.exp(sink[head])), torch.tensor(0.0, dtype=torch.float64)]))
        assert torch.allclose(p[head, 1], e[1] / (e[1].sum() + torch.exp(sink[head])))


def test_plain_choice_within_groups():
    """Four groups of two; group scores 0.3, 0.28, 0.1, 0.05: with two kept groups the second-best expert of all may be
    out of reach of none, and an expert better than a kept one is left out because its group is closed."""
    s = torch.tensor([0.30, 0.01, 0.28, 0.02, 0.10, 0.09, 0.15, 0.05], dtype=torch.float64)
    w = {"p.router": torch.diag(torch.log(s))}
    chosen, weights = plain.route(torch.ones(1, 8, dtype=torch.float64), w, "p.", moe(8, 3, 1, 2.5, (4, 2))["router"])
    assert chosen.tolist() == [[0, 2, 3]]                # 6 (0.15) and 4 (0.10) beat 3 (0.02), but their groups are closed
    want = s[[0, 2, 3]] / s[[0, 2, 3]].sum() * 2.5
    assert torch.allclose(weights[0], want)
    chosen, _ = plain.route(torch.ones(1, 8, dtype=torch.float64), w, "p.", moe(8, 3, 1)["router"])
    assert chosen.tolist() == [[0, 2, 6]]


def test_plain_latent_attention_in_the_latent_space():
    """The plain mixer expands every head's keys and values; scoring the queries against the latents themselves, gating
    what a head mixes and applying the value map afterwards is the same function."""
    m = BAVETAR_A["layers"][1]["mixer"]
    H, D, R, Dv, Q, C, width, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], 64, 31
    g = torch.Generator().manual_seed(5)
    shapes = {"dq": (Q, width), "dq.norm": (Q,), "uq": (H * (D + R), Q), "dkv": (C + R, width), "dkv.norm": (C,), "uk": (H * D, C),
              "uv": (H * Dv, C), "g": (H, width), "sink": (H,), "o": (width, H * Dv)}
    w = {"p." + k: torch.randn(s, generator=g, dtype=torch.float64) * 0.3 for k, s in shapes.items()}
    h = torch.randn(T, width, generator=g, dtype=torch.float64)
    pos = torch.arange(T)
    want = plain.mixer_latent_attention(h, w, "p.", m, 1e-5, pos)
    cq = plain.rms(h @ w["p.dq"].T, 1e-5) * w["p.dq.norm"]
    q = (cq @ w["p.uq"].T).view(T, H, D + R)
    down = h @ w["p.dkv"].T
    c = plain.rms(down[:, :C], 1e-5) * w["p.dkv.norm"]
    qr = plain.rotate_neighbours(q[..., D:], pos, R, m["rot"]["base"])
    kr = plain.rotate_neighbours(down[:, C:], pos, R, m["rot"]["base"])
    ql = torch.einsum("thd,hdc->thc", q[..., :D], w["p.uk"].view(H, D, C))
    scores = (torch.einsum("ihc,jc->hij", ql, c) + torch.einsum("ihr,jr->hij", qr, kr)) * m["scale"]
    mixed = torch.einsum("hij,jc->ihc", plain.softmax_with_sink(scores, w["p.sink"]), c) * torch.sigmoid(h @ w["p.g"].T)[:, :, None]
    got = torch.einsum("ihc,hvc->ihv", mixed, w["p.uv"].view(H, Dv, C)).reshape(T, H * Dv) @ w["p.o"].T
    assert float((got - want).abs().max()) < 1e-10


def test_plain_state_carries_a_prompt():
    """A layer's recurrence over a whole sequence equals itself cut in two with the state handed over by hand."""
    m = mamba(3, 4, 6, 1, 1, 1)["mixer"]
    g = torch.Generator().manual_seed(7)
    T, H, N, Dv = 23, m["heads"], m["state"], m["vdim"]
    x, b, c = (torch.randn(T, H, d, generator=g, dtype=torch.float64) for d in (Dv, N, N))
    dt = torch.rand(T, H, generator=g, dtype=torch.float64)
    rate, skip = torch.ones(H, dtype=torch.float64), torch.zeros(H, dtype=torch.float64)
    whole = plain.state_space_recurrence(x, b, c, dt, rate, skip)
    cut = 9
    S = torch.einsum("sh,sh,shn,shv->hnv", torch.exp(-rate * (dt[:cut].sum(0) - torch.cumsum(dt[:cut], 0))), dt[:cut], b[:cut], x[:cut])
    rest = plain.state_space_recurrence(x[cut:], b[cut:], c[cut:], dt[cut:], rate, skip)
    carried = torch.exp(-rate * torch.cumsum(dt[cut:], 0))[:, :, None] * torch.einsum("hnv,thn->thv", S, c[cut:])
    assert float((rest + carried - whole[cut:]).abs().max()) < 1e-12

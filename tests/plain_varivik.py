"""A plain, slow implementation of the Varivik decoder: one function per mechanism, whole sequences, no cache, no
kernels.  It shares no code with the engine and is what the engine's parts and models are compared with.  ``w`` is a
dict of tensors by checkpoint name, ``cfg`` the contents of config.json.  Everything runs in the type of the tensors
handed in (float64 for a sharp comparison).
"""
import json
import math
import struct
from pathlib import Path

import torch


# ---------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------
def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def turning_rates(dims, base, scaling):
    """Turning rate of pair i, i < dims / 2: base**(-2i/dims).  With ``scaling`` a pair is slowed by ``factor`` where
    its wavelength is longer than original / low, kept where it is shorter than original / high, and blended between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            length = 2.0 * math.pi / f
            low, high, original, factor = (float(scaling[k]) for k in ("low", "high", "original", "factor"))
            if length * low > original:
                f = f / factor
            elif length >= original / high:
                s = (original / length - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_neighbours(x, positions, dims, rates):
    """x [T, heads, dim]: of the first ``dims`` values, 2i and 2i + 1 form a pair that is turned by position * rates[i]."""
    if dims == 0:
        return x
    angle = positions.to(x.dtype)[:, None, None] * torch.tensor(rates, dtype=x.dtype)
    cos, sin = torch.cos(angle), torch.sin(angle)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def visible(T, chunk):
    """[T, T] (query, key): a key not later than the query and, with ``chunk``, of the same chunk."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = j <= i
    return seen if chunk is None else seen & (i // chunk == j // chunk)


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------
def attention(h, w, p, m, positions, v_first):
    """(delta, the values the layer projected and mixed): ``v_first`` is None or what another layer's values are
    blended with."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D)
    k = (h @ w[p + "k"].T).view(T, G, D)
    v = (h @ w[p + "v"].T).view(T, G, Dv)
    rot = m.get("rot")
    if rot is not None:
        rates = turning_rates(rot["dims"], rot["base"], rot.get("scaling"))
        q = rotate_neighbours(q, positions, rot["dims"], rates)
        k = rotate_neighbours(k, positions, rot["dims"], rates)
    if v_first is not None:
        v = mix_values(v, v_first, w[p + "vmix"])
    group = H // G
    scores = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(group, dim=1)) * m["scale"]
    mask = visible(T, m["mask"]["size"] if m.get("mask") else None)
    weights = torch.softmax(scores.masked_fill(~mask, float("-inf")), dim=-1)
    out = torch.einsum("hij,jhd->ihd", weights, v.repeat_interleave(group, dim=1))
    out = out * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return out.reshape(T, H * Dv) @ w[p + "o"].T, v


# ---------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------
def dense(h, w, p):
    gate = h @ w[p + "gate"].T + w[p + "gate.b"]
    up = h @ w[p + "up"].T + w[p + "up.b"]
    return (gelu_tanh(gate) * up) @ w[p + "down"].T + w[p + "down.b"]


def expert(h, w, p):
    return relu_squared(h @ w[p + "up"].T) @ w[p + "down"].T


def route(h, w, p, top):
    """(chosen [T, top], weights [T, top]): softmax over every expert, the largest kept as they are."""
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    best = torch.topk(s, top, dim=-1)
    return best.indices, best.values


def mixture(h, w, p, mlp):
    chosen, weights = route(h, w, p, mlp["router"]["top"])
    rows = []
    for t in range(h.shape[0]):
        row = torch.zeros_like(h[t])
        for e, c in zip(chosen[t].tolist(), weights[t]):
            row = row + c * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
        rows.append(row)
    out = torch.stack(rows)
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return out


def feed_forward(h, w, p, mlp):
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------
def forward(cfg, w, tokens, return_layers=False):
    """logits [T, vocab] of one sequence (and the residual rows behind every layer)."""
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(tokens))
    x = w["embed"][tokens]
    layers, v_first = [], None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mixes = bool(m.get("v_mix"))
        delta, v = attention(rms(x, eps) * w[p + "norm1"], w, p + "mix.", m, positions, v_first if mixes else None)
        if mixes and v_first is None:
            v_first = v
        x = x + delta
        if layer.get("mlp") is not None:
            x = x + feed_forward(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", layer["mlp"])
        layers.append(x.clone())
    logits = (rms(x, eps) * w["final.norm"]) @ w["embed"].T
    return (logits, torch.stack(layers)) if return_layers else logits


def read_folder(folder, dtype=torch.float64):
    """(config.json, tensors by name) of a model folder; bfloat16 and float32 tensors are widened to ``dtype``."""
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    data = raw[8 + n:]
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}
    w = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[info["dtype"]]).view(info["shape"])
        w[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, w


def logits_of(folder, tokens, dtype=torch.float64) -> torch.Tensor:
    cfg, w = read_folder(folder, dtype)
    return forward(cfg, w, tokens)


def greedy(folder, prompt, steps):
    cfg, w = read_folder(folder, torch.float64)
    ids = list(prompt)
    for _ in range(steps):
        ids.append(int(torch.argmax(forward(cfg, w, ids)[-1])))
    return ids[len(prompt):]

"""A plain, slow implementation of the Bavetar decoder: one function per mechanism, whole sequences, no cache, no
kernels, a token-by-token loop where the design is a recurrence.  It shares no code with the engine and is what the
engine's parts and models are compared with.  ``w`` is a dict of tensors by checkpoint name, ``cfg`` the contents of
config.json.  Everything runs in the type of the tensors handed in (float64 for a sharp comparison).
"""
import json
import struct
from pathlib import Path

import torch


# ---------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------
def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    """log(1 + e^x)."""
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def rotate_neighbours(x, positions, dims, base):
    """x [T, ..., dims]: values 2i and 2i + 1 form a pair that is turned by position * base**(-2i/dims)."""
    T = x.shape[0]
    rates = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype)
    angle = positions.to(x.dtype).reshape(T, *([1] * (x.dim() - 1))) * rates
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * torch.cos(angle) - v * torch.sin(angle)
    out[..., 1::2] = v * torch.cos(angle) + u * torch.sin(angle)
    return out


def softmax_with_sink(scores, sink):
    """scores [H, T, T] (query, key): weights over the keys j <= i; the denominator also holds exp(sink_h), a term
    without key or value."""
    T = scores.shape[-1]
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    scores = scores.masked_fill(~seen, float("-inf"))
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def causal_convolution(x, weight, bias):
    """x [T, C], weight [C, taps] (the last column meets the row itself), zeros before the first row; then silu."""
    T, C = x.shape
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x])
    y = torch.zeros_like(x) + bias
    for j in range(taps):
        y = y + padded[j:j + T] * weight[:, j]
    return silu(y)


# ---------------------------------------------------------------------------
# mixers
# ---------------------------------------------------------------------------
def mixer_latent_attention(h, w, p, m, eps, positions):
    """Queries and keys/values through low-rank latents; a rotated key part shared by all heads; a sink per head in
    the softmax; one output gate per head."""
    T = h.shape[0]
    H, D, R, Dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :C], eps) * w[p + "dkv.norm"]
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q_rot = rotate_neighbours(q[..., D:], positions, dims, base)
    k_rot = rotate_neighbours(down[:, C:], positions, dims, base)
    k_plain = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, Dv)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :D], k_plain) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    weights = softmax_with_sink(scores, w[p + "sink"])
    out = torch.einsum("hij,jhd->ihd", weights, v) * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return out.reshape(T, H * Dv) @ w[p + "o"].T


def state_space_recurrence(x, b, c, dt, rate, skip):
    """x [T, H, Dv], b and c [T, H, N], dt [T, H], rate and skip [H]:
    S <- exp(-rate dt_t) S + dt_t b_t x_t^T;  y_t = S^T c_t + skip x_t;  S [N, Dv] starts at zero."""
    T, H, Dv = x.shape
    S = torch.zeros(H, b.shape[-1], Dv, dtype=x.dtype)
    y = torch.empty_like(x)
    for t in range(T):
        S = torch.exp(-rate * dt[t])[:, None, None] * S + (dt[t][:, None] * b[t])[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, c[t]) + skip[:, None] * x[t]
    return y


def mixer_mamba2(h, w, p, m, eps, stored=lambda t: t):
    """``stored``: what is done to the projected rows (without the step sizes) and to the convolved rows between two steps
    of the computation -- nothing, or a rounding to the type they are kept in."""
    T = h.shape[0]
    H, Dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * Dv
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    z, xbc = stored(z), stored(xbc)
    xbc = stored(causal_convolution(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, b, c = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    per = H // G
    b = b.reshape(T, G, N).repeat_interleave(per, dim=1)
    c = c.reshape(T, G, N).repeat_interleave(per, dim=1)
    dt = softplus(dt + w[p + "dt_bias"])
    y = state_space_recurrence(x.reshape(T, H, Dv), b, c, dt, torch.exp(w[p + "A_log"]), w[p + "D"])
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def mixer(kind, h, w, p, m, eps, positions):
    if kind == "latent_attention":
        return mixer_latent_attention(h, w, p, m, eps, positions)
    if kind == "mamba2":
        return mixer_mamba2(h, w, p, m, eps)
    raise ValueError(f"unknown mixer {kind!r}")


# ---------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------
def dense(h, w, p):
    u = torch.clamp(h @ w[p + "up"].T, min=0.0)
    return (u * u) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, router):
    """(chosen [T, top], weights [T, top]): softmax over all experts; only experts of the ``keep`` groups with the
    largest best score may be chosen; the weights are the chosen scores over their sum, times ``scale``."""
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    groups = router.get("groups")
    choice = s
    if groups is not None:
        best = s.view(s.shape[0], groups["count"], -1).max(-1).values
        kept = torch.zeros_like(best).scatter_(1, torch.topk(best, groups["keep"], dim=-1).indices, 1.0)
        open_ = kept.repeat_interleave(s.shape[1] // groups["count"], dim=1) > 0
        choice = s.masked_fill(~open_, -1.0)
    chosen = torch.topk(choice, router["top"], dim=-1).indices
    weights = torch.gather(s, 1, chosen)
    weights = weights / (weights.sum(-1, keepdim=True) + 1e-20) * router.get("scale", 1.0)
    return chosen, weights


def mixture(h, w, p, mlp):
    chosen, weights = route(h, w, p, mlp["router"])
    out = torch.zeros_like(h)
    for e in sorted(set(chosen.flatten().tolist())):
        rows, which = torch.nonzero(chosen == e, as_tuple=True)
        out[rows] += weights[rows, which][:, None] * expert(h[rows], w, f"{p}e{e}.")
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
    layers = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        delta = mixer(layer["type"], rms(x, eps) * w[p + "norm1"], w, p + "mix.", layer["mixer"], eps, positions)
        if layer.get("mlp") is not None:
            delta = delta + feed_forward(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", layer["mlp"])
        x = x + delta
        layers.append(x.clone())
    y = rms(x, eps) * w["final.norm"]
    logits = (y @ w["embed"].T) * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(layers)) if return_layers else logits


def read_folder(folder, dtype=torch.float64):
    """(config.json, tensors by name) of a model folder; floating-point tensors are widened to ``dtype``."""
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
        t = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[info["dtype"]]).view(*info["shape"])
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

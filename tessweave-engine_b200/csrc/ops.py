"""Python side of the CUDA kernels: thin launch wrappers over the compiled libraries.

Each wrapper checks what the kernel assumes (device, element type, contiguity,
sizes it can take) and raises a clear error otherwise; a kernel is never handed
a shape it would compute wrongly.  There is no fallback: if a library cannot be
compiled or loaded, the call fails.  Launches go to torch's current stream, so
they order with library matrix products and can be captured in CUDA graphs.
"""
from __future__ import annotations

import ctypes
from ctypes import c_void_p, c_int, c_float, c_long
from dataclasses import dataclass

import torch

from .build import load_library

F32, BF16 = 0, 1


class KernelError(RuntimeError):
    pass


@dataclass
class SplitSum:
    """The result of a matrix product that was split over k: fp32 slices [slices, rows, width]
    whose sum (in slice order) is the product.  Kernels that consume it add the slices
    themselves; ``dense()`` adds them for anyone else."""
    slices: torch.Tensor

    def dense(self, dtype: torch.dtype, out: torch.Tensor | None = None) -> torch.Tensor:
        n, rows, width = self.slices.shape
        out = out if out is not None else torch.empty(rows, width, dtype=dtype, device=self.slices.device)
        code = _fn("gemm_smallm", "tw_reduce_partial")(_ptr(out), _ptr(self.slices), c_int(n), c_long(rows * width),
                                                       c_int(dtype_code(dtype)), _stream())
        _check(code, "reduce_partial")
        return out


def dtype_code(dtype: torch.dtype) -> int:
    if dtype == torch.float32:
        return F32
    if dtype == torch.bfloat16:
        return BF16
    raise KernelError(f"kernels take float32 or bfloat16 activations, not {dtype}")


def _ptr(t: torch.Tensor | None) -> c_void_p:
    return c_void_p(0 if t is None else t.data_ptr())


def _stream() -> c_void_p:
    # the raw handle of torch's current stream (what torch.cuda.current_stream().cuda_stream gives, without
    # building a Stream object for every launch)
    return c_void_p(torch._C._cuda_getCurrentRawStream(torch.cuda.current_device()))


def _need(cond: bool, message: str) -> None:
    if not cond:
        raise KernelError(message)


def _cuda(*tensors: torch.Tensor | None) -> None:
    for t in tensors:
        if t is not None and not t.is_cuda:
            raise KernelError("kernel operands must live on a CUDA device; this engine has no CPU path")


def _check(code: int, what: str) -> None:
    if code != 0:
        raise KernelError(f"{what}: CUDA error {code} at launch "
                          f"({torch.cuda.get_device_name() if torch.cuda.is_available() else 'no device'})")


_sigs_done: set[str] = set()
LAUNCHES = [0]      # kernel launchers called so far (each call launches at least one kernel)
CALL_LOG: list[str] | None = None     # when a list: the launchers called, by name (who measures asks which kernel ran)


def note_call(name: str) -> None:
    if CALL_LOG is not None:
        CALL_LOG.append(name)


def _fn(lib_name: str, fn_name: str, defines=None):
    LAUNCHES[0] += 1
    note_call(fn_name)
    lib = load_library(lib_name, defines)
    fn = getattr(lib, fn_name)
    key = f"{lib_name}:{fn_name}:{defines}"
    if key not in _sigs_done:
        fn.restype = c_int
        _sigs_done.add(key)
    return fn


# ---------------------------------------------------------------------------
def embed(resid: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, n_tokens: int, status: torch.Tensor,
          device_tokens: torch.Tensor | None = None, scale: float = 1.0) -> None:
    """resid[n] = float(table[ids[n]]) * scale; resid is fp32 [>=n_tokens, hidden].  An id -(i + 1) is
    replaced by ``device_tokens[i]`` (int32, on the device) inside the kernel."""
    _cuda(resid, table, ids, status, device_tokens)
    _need(device_tokens is None or device_tokens.dtype == torch.int32, "embed: device tokens must be int32")
    _need(resid.dtype == torch.float32 and resid.is_contiguous(), "embed: residual stream must be contiguous fp32")
    _need(table.is_contiguous() and ids.dtype == torch.int32, "embed: table contiguous, ids int32")
    _need(resid.shape[0] >= n_tokens and ids.numel() >= n_tokens and resid.shape[1] == table.shape[1],
          "embed: shapes disagree")
    code = _fn("elementwise", "tw_embed")(_ptr(resid), _ptr(table), _ptr(ids), _ptr(device_tokens),
                                          c_int(0 if device_tokens is None else device_tokens.numel()), c_int(n_tokens),
                                          c_int(table.shape[1]), c_int(table.shape[0]), c_float(scale),
                                          c_int(dtype_code(table.dtype)), _ptr(status), _stream())
    _check(code, "embed")


def rmsnorm_to_residual(resid: torch.Tensor, delta, weight: torch.Tensor, eps: float, n_rows: int,
                        copy: torch.Tensor | None = None) -> None:
    """resid += rmsnorm(delta) * weight (in place, fp32 statistics and sum); ``copy`` (may be None) receives the
    new rows in its own type, for the product that reads them next.  ``delta`` is a tensor of the
    activation type (the type of ``copy``; fp32 where there is no copy) or a ``SplitSum``."""
    partial, nsplit, split_stride = None, 0, 0
    hidden = resid.shape[1]
    if isinstance(delta, SplitSum):
        partial, nsplit, split_stride = delta.slices, delta.slices.shape[0], delta.slices.stride(0)
        _need(partial.dtype == torch.float32 and partial.shape[2] == hidden and partial[0].is_contiguous()
              and partial.shape[1] >= n_rows, "rmsnorm_to_residual: split sum must be fp32 [slices, rows, hidden]")
        delta = None
    _cuda(resid, delta, weight, copy, partial)
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and resid.shape[0] >= n_rows,
          "rmsnorm_to_residual: residual stream must be contiguous fp32")
    _need(weight.dtype == torch.float32 and weight.numel() == hidden, "rmsnorm_to_residual: weight must be fp32 [hidden]")
    dtype = copy.dtype if copy is not None else (delta.dtype if delta is not None else torch.float32)
    if copy is not None:
        _need(copy.is_contiguous() and copy.shape[1] == hidden and copy.shape[0] >= n_rows, "rmsnorm_to_residual: bad copy")
    if delta is not None:
        _need(delta.dtype == dtype and delta.is_contiguous() and delta.shape[1] == hidden and delta.shape[0] >= n_rows,
              "rmsnorm_to_residual: delta must be contiguous [rows, hidden] of the activation type")
    code = _fn("elementwise", "tw_rmsnorm_to_residual")(_ptr(resid), _ptr(copy), _ptr(delta), _ptr(partial), c_int(nsplit),
                                                        c_long(split_stride), _ptr(weight), c_float(eps), c_int(n_rows),
                                                        c_int(hidden), c_int(dtype_code(dtype)), _stream())
    _check(code, "rmsnorm_to_residual")


def round_rows(out: torch.Tensor, resid: torch.Tensor, n_rows: int) -> None:
    """out[:n_rows] = resid[:n_rows] in the type of ``out``."""
    _cuda(out, resid)
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and out.is_contiguous()
          and out.shape[1] == resid.shape[1] and min(out.shape[0], resid.shape[0]) >= n_rows, "round_rows: bad operands")
    code = _fn("elementwise", "tw_round_rows")(_ptr(out), _ptr(resid), c_long(n_rows * resid.shape[1]),
                                               c_int(dtype_code(out.dtype)), _stream())
    _check(code, "round_rows")


# ---------------------------------------------------------------------------
# sigmoid attention with mixed heads (csrc/sigmoid_attention.cu)
# ---------------------------------------------------------------------------
def sigmoid_attention_prepare(qf: torch.Tensor, proj: torch.Tensor, q_norm_w: torch.Tensor, k_norm_w: torch.Tensor,
                              eps: float, mix: torch.Tensor | None, scale: float, inv_freq: torch.Tensor | None,
                              rot_dims: int, interleaved: bool, positions: torch.Tensor, seq_of_token: torch.Tensor,
                              seq_slot: torch.Tensor, block_table: torch.Tensor, k_pages: torch.Tensor,
                              v_pages: torch.Tensor, n_tokens: int, n_q_heads: int, n_kv_heads: int, head_dim: int,
                              write_cache: bool, status: torch.Tensor) -> None:
    """Per token: norms over the whole q and k projections, rotation, the raw key into the value pages, the
    normalised rotated key into the key pages, the folded query ``qf`` [rows, Hq, Hkv * D] (the heads' mixing
    matrix ``mix`` [Hq, Hq] and ``scale`` applied).  ``proj`` rows are [q | k | anything]."""
    _cuda(qf, proj, q_norm_w, k_norm_w, mix, inv_freq, positions, seq_of_token, seq_slot, block_table, k_pages, v_pages, status)
    qw, kw = n_q_heads * head_dim, n_kv_heads * head_dim
    _need(proj.stride(1) == 1 and proj.shape[1] >= qw + kw and proj.shape[0] >= n_tokens, "sigmoid attention: bad projection rows")
    _need(qf.is_contiguous() and qf.dtype == proj.dtype and qf.numel() >= n_tokens * n_q_heads * kw,
          "sigmoid attention: folded queries must be contiguous [rows, Hq, Hkv * D] of the activation type")
    _need(q_norm_w.dtype == torch.float32 and q_norm_w.numel() == qw and k_norm_w.dtype == torch.float32
          and k_norm_w.numel() == kw, "sigmoid attention: norm weights must be fp32 [Hq * D] and [Hkv * D]")
    if mix is not None:
        _need(mix.dtype == torch.float32 and mix.is_contiguous() and tuple(mix.shape) == (n_q_heads, n_q_heads),
              "sigmoid attention: the mixing matrix must be fp32 [Hq, Hq]")
    if inv_freq is not None:
        _need(inv_freq.dtype == torch.float32 and inv_freq.numel() == rot_dims // 2 and rot_dims % 2 == 0
              and rot_dims <= head_dim, "sigmoid attention: inv_freq must be fp32 [rot_dims / 2], rot_dims even and <= D")
    _need(k_pages.dtype == proj.dtype and v_pages.dtype == proj.dtype and k_pages.is_contiguous() and v_pages.is_contiguous()
          and tuple(k_pages.shape[1:]) == (n_kv_heads, k_pages.shape[2], head_dim) and v_pages.shape == k_pages.shape,
          "sigmoid attention: cache pages must be contiguous [pages, kv_heads, page, head_dim] of the activation type")
    _need(block_table.dtype == torch.int32 and block_table.dim() == 2 and block_table.is_contiguous(),
          "sigmoid attention: block table must be contiguous int32 [requests, blocks]")
    code = _fn("sigmoid_attention", "tw_sigattn_prepare")(
        _ptr(proj), c_int(proj.stride(0)), _ptr(q_norm_w), _ptr(k_norm_w), c_float(eps), _ptr(mix), c_float(scale),
        _ptr(inv_freq), c_int(rot_dims if inv_freq is not None else 0), c_int(1 if interleaved else 0), _ptr(positions),
        _ptr(seq_of_token), _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(qf), _ptr(k_pages),
        _ptr(v_pages), c_int(n_tokens), c_int(n_q_heads), c_int(n_kv_heads), c_int(head_dim), c_int(k_pages.shape[2]),
        c_int(k_pages.shape[0]), c_int(1 if write_cache else 0), c_int(dtype_code(proj.dtype)), _ptr(status), _stream())
    _check(code, "sigmoid_attention_prepare")


def sigmoid_attention_generic(out: torch.Tensor, qf: torch.Tensor, bias: torch.Tensor | None, gate: torch.Tensor | None,
                              positions: torch.Tensor, seq_of_token: torch.Tensor, seq_slot: torch.Tensor,
                              block_table: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, n_tokens: int,
                              n_q_heads: int, n_kv_heads: int, head_dim: int, window: int, status: torch.Tensor) -> None:
    """Exact paged causal sigmoid attention, one block per (token, head): out[n, h] = sum over visible keys of
    sigmoid(qf[n, h] . k + bias[h]) * v, then * sigmoid(gate[n, h]) where a gate is given (a column slice of
    the projection buffer is fine: its row stride is passed on)."""
    _cuda(out, qf, bias, gate, positions, seq_of_token, seq_slot, block_table, k_pages, v_pages, status)
    _need(head_dim <= 256 and n_q_heads % n_kv_heads == 0, "sigmoid attention: head_dim above 256 or bad head counts")
    _need(out.stride(1) == 1 and qf.is_contiguous() and qf.dtype == out.dtype == k_pages.dtype, "sigmoid attention: bad operands")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == n_q_heads), "sigmoid attention: bias must be fp32 [Hq]")
    _need(gate is None or (gate.dtype == out.dtype and gate.stride(1) == 1 and gate.shape[1] >= n_q_heads * head_dim),
          "sigmoid attention: gate must be [rows, Hq * D] of the activation type")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "sigmoid attention: bad block table")
    code = _fn("sigmoid_attention", "tw_sigattn_generic")(
        _ptr(out), c_int(out.stride(0)), _ptr(qf), _ptr(bias), _ptr(gate), c_int(0 if gate is None else gate.stride(0)),
        _ptr(positions), _ptr(seq_of_token), _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages),
        _ptr(v_pages), c_int(n_tokens), c_int(n_q_heads), c_int(n_kv_heads), c_int(head_dim), c_int(k_pages.shape[2]),
        c_int(k_pages.shape[0]), c_int(window), c_int(dtype_code(out.dtype)), _ptr(status), _stream())
    _check(code, "sigmoid_attention_generic")


def sigmoid_attention_tensor_cores(dtype: torch.dtype, head_dim: int, n_kv_heads: int) -> bool:
    """Whether the tensor-core kernels (csrc/sigmoid_attention_bf16.cu) take the shape: bfloat16, a head size that is a
    multiple of 16 up to 256, and a tile of 64 folded queries plus the ring of four key chunks within 227 KB of shared
    memory.  TESSWEAVE_SIGMOID_ATTENTION=exact sends everything to the exact kernel."""
    import os
    if os.environ.get("TESSWEAVE_SIGMOID_ATTENTION") == "exact":
        return False
    if dtype != torch.bfloat16 or head_dim % 16 or not 16 <= head_dim <= 256:
        return False
    return 64 * (n_kv_heads * head_dim + 8) * 2 + 4 * 64 * (head_dim + 8) * 2 <= 227 * 1024


def sigmoid_decode_heads_per_block() -> int:
    """0: a block of the sliced-keys kernel serves up to 32 heads of a request (the keys are read once for all of
    them); TESSWEAVE_SIGMOID_DECODE_HEADS=16 forces blocks of 16 heads (half the registers, the keys read twice)."""
    import os
    return 16 if os.environ.get("TESSWEAVE_SIGMOID_DECODE_HEADS") == "16" else 0


def sigmoid_decode_splits(n_seqs: int, n_heads: int, max_kv_len: int) -> int:
    """Slices a single token's keys are cut into: enough blocks (request x up to 32 heads x slice) for two per SM,
    at least one tile of 64 keys per slice, at most 64 slices.  A block streams its slice slowly (it waits on its own
    chain of dependent tensor-core products), so the bandwidth comes from the number of blocks: one request with 4,096
    keys takes 24 us with 32 slices and 18 us with 64."""
    import os
    forced = os.environ.get("TESSWEAVE_SIGMOID_DECODE_SPLITS")
    tiles = max(1, -(-max_kv_len // 64))
    if forced:
        return max(1, min(int(forced), 64, tiles))
    groups = max(1, n_seqs * -(-n_heads // (32 if n_heads > 16 and not sigmoid_decode_heads_per_block() else 16)))
    return max(1, min((2 * _SM_COUNT) // groups, tiles, 64))


def _sigattn_checks(out, qf, bias, gate, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim):
    _cuda(out, qf, bias, gate, block_table, k_pages, v_pages)
    _need(out.dtype == torch.bfloat16 and qf.dtype == torch.bfloat16 and k_pages.dtype == torch.bfloat16
          and v_pages.dtype == torch.bfloat16, "sigmoid attention (tensor cores): operands must be bfloat16")
    _need(out.stride(1) == 1 and qf.is_contiguous() and qf.data_ptr() % 16 == 0, "sigmoid attention: bad out / folded queries")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and v_pages.shape == k_pages.shape
          and tuple(k_pages.shape[1:]) == (n_kv_heads, k_pages.shape[2], head_dim) and k_pages.data_ptr() % 16 == 0
          and v_pages.data_ptr() % 16 == 0, "sigmoid attention: cache pages must be contiguous [pages, kv_heads, page, head_dim]")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == n_q_heads), "sigmoid attention: bias must be fp32 [Hq]")
    _need(gate is None or (gate.dtype == torch.bfloat16 and gate.stride(1) == 1 and gate.shape[1] >= n_q_heads * head_dim
                           and gate.data_ptr() % 4 == 0 and gate.stride(0) % 2 == 0),
          "sigmoid attention: gate must be bfloat16 [rows, Hq * D]")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "sigmoid attention: bad block table")
    _need(n_q_heads % n_kv_heads == 0, "sigmoid attention: query heads must be a multiple of key/value heads")


def sigmoid_attention_prefill(out, qf, bias, gate, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages,
                              v_pages, n_seqs: int, max_q_len: int, n_q_heads: int, n_kv_heads: int, head_dim: int,
                              window: int, skip_singles: bool, status: torch.Tensor) -> None:
    """Tensor-core sigmoid attention for the requests of a step that bring several tokens (and, unless
    ``skip_singles``, those that bring one): out[row, h] = (sum of sigmoid(qf . k + bias) v) * sigmoid(gate)."""
    _sigattn_checks(out, qf, bias, gate, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim)
    code = _fn("sigmoid_attention_bf16", "tw_sigattn_prefill", {"TW_HEAD_DIM": head_dim})(
        _ptr(out), c_int(out.stride(0)), _ptr(qf), _ptr(bias), _ptr(gate), c_int(0 if gate is None else gate.stride(0)),
        _ptr(seq_q_start), _ptr(seq_q_len), _ptr(seq_kv_len), _ptr(seq_slot), _ptr(block_table),
        c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(n_seqs), c_int(max_q_len), c_int(n_q_heads),
        c_int(n_kv_heads), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]), c_int(window), c_int(1 if skip_singles else 0),
        _ptr(status), _stream())
    _check(code, "sigmoid_attention_prefill")


SIGMOID_TCGEN05_MIN_TOKENS = 128


def sigmoid_tcgen05_key_tile() -> int:
    """Keys per tile of the tcgen05 sigmoid attention: 128, or 64 with TESSWEAVE_SIGMOID_KEY_TILE=64 (chunks of 64
    keys make the rings beside the folded queries twice as deep, but a tile's fixed costs come twice as often:
    measured 226 us against 199 us for 2,048 tokens at 28 heads, 4 key/value heads of 128)."""
    import os
    return 64 if os.environ.get("TESSWEAVE_SIGMOID_KEY_TILE") == "64" else 128


def sigmoid_attention_tcgen05(dtype: torch.dtype, head_dim: int, n_kv_heads: int, page_size: int, max_q_len: int) -> bool:
    """Whether a step whose longest portion has ``max_q_len`` tokens runs its sigmoid attention on the tcgen05 kernel
    (csrc/sigmoid_attention_tcgen05.cu): bfloat16, head size 64 or 128, pages that divide a tile of 64 keys or are a
    multiple of it, folded queries of 128 rows that leave room for three chunks of keys in shared memory, and a
    portion of at least 128 tokens.  TESSWEAVE_SIGMOID_PREFILL=mma|tcgen05 forces one of the two (the latter only
    for shapes the kernel takes)."""
    import os
    if dtype != torch.bfloat16 or head_dim not in (64, 128) or page_size < 4:
        return False
    tile = sigmoid_tcgen05_key_tile()
    if not (tile % page_size == 0 or page_size % tile == 0):
        return False
    blocks = head_dim // 64
    if (227 * 1024 - 1024 - 512 - n_kv_heads * blocks * 16384) // (blocks * tile * 128) < 3:
        return False
    forced = os.environ.get("TESSWEAVE_SIGMOID_PREFILL")
    if forced == "mma":
        return False
    if forced == "tcgen05":
        return True
    return max_q_len >= SIGMOID_TCGEN05_MIN_TOKENS


def sigmoid_attention_prefill_tcgen05(out, qf, bias, gate, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table,
                                      k_pages, v_pages, n_seqs: int, max_q_len: int, n_q_heads: int, n_kv_heads: int,
                                      head_dim: int, window: int, skip_singles: bool, status: torch.Tensor) -> None:
    """The same as ``sigmoid_attention_prefill`` on the 5th-generation tensor cores (TMA, tcgen05.mma, S and O in
    tensor memory), for the shapes ``sigmoid_attention_tcgen05`` names."""
    _sigattn_checks(out, qf, bias, gate, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim)
    _need(out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0, "tcgen05 sigmoid attention: rows of out must be 16-byte aligned")
    _need(gate is None or (gate.data_ptr() % 16 == 0 and gate.stride(0) % 8 == 0),
          "tcgen05 sigmoid attention: rows of the gate must be 16-byte aligned")
    code = _fn("sigmoid_attention_tcgen05", "tw_sigattn_prefill_tc5",
               {"TW_HEAD_DIM": head_dim, "TW_SIG_KEY_TILE": sigmoid_tcgen05_key_tile()})(
        _ptr(out), c_int(out.stride(0)), _ptr(qf), _ptr(bias), _ptr(gate), c_int(0 if gate is None else gate.stride(0)),
        _ptr(seq_q_start), _ptr(seq_q_len), _ptr(seq_kv_len), _ptr(seq_slot), _ptr(block_table),
        c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(n_seqs), c_int(max_q_len), c_int(n_q_heads),
        c_int(n_kv_heads), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]), c_int(window), c_int(1 if skip_singles else 0),
        _ptr(status), _stream())
    _check(code, "sigmoid_attention_prefill_tcgen05")


def sigmoid_attention_decode(out, partial, qf, bias, gate, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table,
                             k_pages, v_pages, n_seqs: int, n_q_heads: int, n_kv_heads: int, head_dim: int, window: int,
                             nsplit: int, status: torch.Tensor) -> None:
    """Tensor-core sigmoid attention for the requests of a step that bring one token, their keys cut into
    ``nsplit`` slices; ``partial`` is fp32 scratch of at least n_seqs * nsplit * Hq * D values."""
    _sigattn_checks(out, qf, bias, gate, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim)
    _need(partial.dtype == torch.float32 and partial.is_contiguous()
          and partial.numel() >= n_seqs * nsplit * n_q_heads * head_dim and 1 <= nsplit <= 64,
          "sigmoid attention: scratch must be fp32 [requests, slices, Hq, D], 1 to 64 slices")
    code = _fn("sigmoid_attention_bf16", "tw_sigattn_decode", {"TW_HEAD_DIM": head_dim})(
        _ptr(out), c_int(out.stride(0)), _ptr(partial), _ptr(qf), _ptr(bias), _ptr(gate),
        c_int(0 if gate is None else gate.stride(0)), _ptr(seq_q_start), _ptr(seq_q_len), _ptr(seq_kv_len), _ptr(seq_slot),
        _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(n_seqs), c_int(n_q_heads),
        c_int(n_kv_heads), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]), c_int(window), c_int(nsplit),
        c_int(sigmoid_decode_heads_per_block()), _ptr(status), _stream())
    _check(code, "sigmoid_attention_decode")


# ---------------------------------------------------------------------------
# gated recurrences with a fixed-size state per request (csrc/recurrent.cu)
# ---------------------------------------------------------------------------
def mingru_scan(out: torch.Tensor, proj: torch.Tensor, bias_z: torch.Tensor | None, bias_x: torch.Tensor | None,
                state: torch.Tensor, seq_slot: torch.Tensor, seq_q_start: torch.Tensor, seq_q_len: torch.Tensor,
                n_seqs: int, max_q_len: int, width: int, write_state: bool = True) -> None:
    """Rows of ``proj`` are [z | x | g] pre-activations (each ``width`` wide); for every request of the step the
    state S (fp32 [slots, width], row ``seq_slot``) runs through its rows: S = (1 - z) S + z c, and
    out = S * silu(g) in the type of ``out``.  ``max_q_len`` (the longest portion of the step) chooses between one
    thread per channel and a block that cuts a long portion into segments."""
    _cuda(out, proj, bias_z, bias_x, state, seq_slot, seq_q_start, seq_q_len)
    _need(proj.stride(1) == 1 and proj.shape[1] >= 3 * width and out.stride(1) == 1 and out.shape[1] >= width
          and out.dtype == proj.dtype, "mingru: rows must be [z | x | g] and the output of the same type")
    _need(state.dtype == torch.float32 and state.is_contiguous() and state.shape[1] == width, "mingru: state must be fp32 [slots, width]")
    for b in (bias_z, bias_x):
        _need(b is None or (b.dtype == torch.float32 and b.numel() == width), "mingru: biases must be fp32 [width]")
    code = _fn("recurrent", "tw_mingru_scan")(
        _ptr(out), c_int(out.stride(0)), _ptr(proj), c_int(proj.stride(0)), _ptr(bias_z), _ptr(bias_x), _ptr(state),
        _ptr(seq_slot), _ptr(seq_q_start), _ptr(seq_q_len), c_int(n_seqs), c_int(max_q_len), c_int(width),
        c_int(1 if write_state else 0),
        c_int(dtype_code(out.dtype)), _stream())
    _check(code, "mingru_scan")


def add_rmsnorm(out: torch.Tensor, resid: torch.Tensor, delta, weight: torch.Tensor,
                eps: float, n_rows: int, rows: torch.Tensor | None = None, delta_scale: float = 1.0) -> None:
    """resid += delta_scale * delta (in place, fp32) and out = rmsnorm(resid) * weight.

    ``delta`` is None, a tensor of the output's type, or a ``SplitSum`` (fp32 slices of a
    matrix product split over k, added here in slice order).  With ``rows`` (int32 indices)
    only those rows are normalised, into out[0..n_rows), and the residual stream is left
    as it was.
    """
    partial, nsplit, split_stride = None, 0, 0
    if isinstance(delta, SplitSum):
        partial, nsplit, split_stride = delta.slices, delta.slices.shape[0], delta.slices.stride(0)
        _need(partial.dtype == torch.float32 and partial.shape[2] == resid.shape[1] and partial[0].is_contiguous(),
              "rmsnorm: split sum must be fp32 [slices, rows, hidden]")
        delta = None
    _cuda(out, resid, delta, weight, rows, partial)
    hidden = resid.shape[1]
    _need(resid.dtype == torch.float32 and resid.is_contiguous(), "rmsnorm: residual stream must be contiguous fp32")
    _need(weight.dtype == torch.float32 and weight.numel() == hidden, "rmsnorm: weight must be fp32 [hidden]")
    _need(out.is_contiguous() and out.shape[1] == hidden and out.shape[0] >= n_rows, "rmsnorm: bad output")
    if delta is not None:
        _need(delta.dtype == out.dtype and delta.is_contiguous() and delta.shape[1] == hidden,
              "rmsnorm: delta must match the output type and width")
    if rows is not None:
        _need(rows.dtype == torch.int32 and rows.numel() >= n_rows, "rmsnorm: rows must be int32")
    else:
        _need(resid.shape[0] >= n_rows, "rmsnorm: fewer residual rows than asked")
    code = _fn("elementwise", "tw_add_rmsnorm")(_ptr(out), _ptr(resid), _ptr(delta), _ptr(partial), c_int(nsplit),
                                                c_long(split_stride), _ptr(weight), c_float(eps),
                                                c_int(n_rows), c_int(hidden), _ptr(rows), c_float(delta_scale),
                                                c_int(dtype_code(out.dtype)), _stream())
    _check(code, "add_rmsnorm")


def _delta_operand(delta, like: torch.Tensor, hidden: int, n_rows: int | None, what: str):
    """(tensor or None, slices or None, number of slices, their stride) of a delta that a norm kernel adds."""
    if isinstance(delta, SplitSum):
        slices = delta.slices
        _need(slices.dtype == torch.float32 and slices.shape[2] == hidden and slices[0].is_contiguous(),
              f"{what}: split sum must be fp32 [slices, rows, hidden]")
        return None, slices, slices.shape[0], slices.stride(0)
    _need(delta is None or (delta.dtype == like.dtype and delta.is_contiguous() and delta.shape[1] == hidden
                            and (n_rows is None or delta.shape[0] >= n_rows)), f"{what}: delta must match the output type and width")
    return delta, None, 0, 0


def add_rmsnorm_pair(out: torch.Tensor, out2: torch.Tensor | None, resid: torch.Tensor, delta, delta2, weight: torch.Tensor,
                     weight2: torch.Tensor | None, eps: float, n_rows: int, rows: torch.Tensor | None = None,
                     delta_scale: float = 1.0) -> None:
    """resid += delta_scale * (delta + delta2) (in place, fp32), out = rmsnorm(resid) * weight and out2 = rmsnorm(resid) *
    weight2: what a layer whose two sub-layers read one stream through norms of their own does between layers.  Each
    delta as in ``add_rmsnorm`` and either may be None; ``out2`` None: one result.  ``rows`` as in ``add_rmsnorm``."""
    hidden = resid.shape[1]
    n_src = None if rows is not None else n_rows
    d1, p1, n1, s1 = _delta_operand(delta, out, hidden, n_src, "rmsnorm pair")
    d2, p2, n2, s2 = _delta_operand(delta2, out, hidden, n_src, "rmsnorm pair")
    _cuda(out, out2, resid, d1, p1, d2, p2, weight, weight2, rows)
    _need(resid.dtype == torch.float32 and resid.is_contiguous(), "rmsnorm pair: residual stream must be contiguous fp32")
    _need((out2 is None) == (weight2 is None), "rmsnorm pair: a second result has a weight of its own")
    for o, w in ((out, weight), (out2, weight2)):
        _need(o is None or (o.is_contiguous() and o.dtype == out.dtype and o.shape[1] == hidden and o.shape[0] >= n_rows
                            and w.dtype == torch.float32 and w.numel() == hidden and w.is_contiguous()),
              "rmsnorm pair: results of one type and the stream's width, with fp32 weights")
    if rows is not None:
        _need(rows.dtype == torch.int32 and rows.numel() >= n_rows, "rmsnorm pair: rows must be int32")
    else:
        _need(resid.shape[0] >= n_rows, "rmsnorm pair: fewer residual rows than asked")
    code = _fn("elementwise", "tw_add_rmsnorm_pair")(
        _ptr(out), _ptr(out2), _ptr(resid), _ptr(d1), _ptr(p1), c_int(n1), c_long(s1), _ptr(d2), _ptr(p2), c_int(n2), c_long(s2),
        _ptr(weight), _ptr(weight2), c_float(eps), c_int(n_rows), c_int(hidden), _ptr(rows), c_float(delta_scale),
        c_int(dtype_code(out.dtype)), _stream())
    _check(code, "add_rmsnorm_pair")


def rope_kv_write(qkv: torch.Tensor, bias: torch.Tensor | None, positions: torch.Tensor, seq_of_token: torch.Tensor,
                  seq_slot: torch.Tensor, block_table: torch.Tensor, inv_freq: torch.Tensor | None,
                  k_pages: torch.Tensor, v_pages: torch.Tensor, n_tokens: int, n_q_heads: int, n_kv_heads: int,
                  head_dim: int, write_cache: bool, status: torch.Tensor, source: "SplitSum | None" = None) -> None:
    """Add the bias, rotate q and k by position, store k and v in their cache pages.

    qkv: [>=n_tokens, (Hq + 2 Hkv) * D]; k_pages/v_pages: [pages, Hkv, page, D].  With
    ``source`` the projection is read from the fp32 slices of a split product instead of
    ``qkv``; the rotated q is written to ``qkv`` either way.
    """
    _cuda(qkv, bias, positions, seq_of_token, seq_slot, block_table, inv_freq, k_pages, v_pages, status)
    width = (n_q_heads + 2 * n_kv_heads) * head_dim
    partial, nsplit, split_stride = None, 0, 0
    if source is not None:
        partial, nsplit, split_stride = source.slices, source.slices.shape[0], source.slices.stride(0)
        _need(partial.is_cuda and partial.dtype == torch.float32 and partial.shape[2] == width
              and partial[0].is_contiguous() and partial.shape[1] >= n_tokens, "rope: bad split source")
    _need(qkv.stride(1) == 1 and qkv.shape[1] == width, "rope: qkv row must be [q | k | v] heads")
    _need(head_dim % 2 == 0, f"rope: head_dim {head_dim} must be even")
    _need(k_pages.dtype == qkv.dtype and v_pages.dtype == qkv.dtype and k_pages.is_contiguous()
          and v_pages.is_contiguous(), "rope: cache pages must be contiguous and of the activation type")
    _need(tuple(k_pages.shape[1:]) == (n_kv_heads, k_pages.shape[2], head_dim) and v_pages.shape == k_pages.shape,
          "rope: cache pages must be [pages, kv_heads, page, head_dim]")
    _need(block_table.dtype == torch.int32 and block_table.dim() == 2 and block_table.is_contiguous(),
          "rope: block table must be contiguous int32 [requests, blocks]")
    if bias is not None:
        _need(bias.dtype == torch.float32 and bias.numel() == width, "rope: bias must be fp32 [(Hq+2Hkv)*D]")
    if inv_freq is not None:
        _need(inv_freq.dtype == torch.float32 and inv_freq.numel() == head_dim // 2, "rope: inv_freq must be fp32 [D/2]")
    code = _fn("elementwise", "tw_rope_kv_write")(
        _ptr(qkv), c_int(qkv.stride(0)), _ptr(partial), c_int(nsplit), c_long(split_stride), _ptr(bias),
        _ptr(positions), _ptr(seq_of_token), _ptr(seq_slot),
        _ptr(block_table), c_int(block_table.shape[1]), _ptr(inv_freq), _ptr(k_pages), _ptr(v_pages),
        c_int(n_tokens), c_int(n_q_heads), c_int(n_kv_heads), c_int(head_dim), c_int(k_pages.shape[2]),
        c_int(k_pages.shape[0]), c_int(1 if write_cache else 0), c_int(dtype_code(qkv.dtype)), _ptr(status), _stream())
    _check(code, "rope_kv_write")


def rotate_heads(rows: torch.Tensor, bias: torch.Tensor | None, positions: torch.Tensor, seq_of_token: torch.Tensor,
                 inv_freq: torch.Tensor | None, n_tokens: int, n_heads: int, head_dim: int) -> None:
    """In place on the first ``n_heads`` heads of each packed row: add the bias, then rotate
    by position (either may be absent).  Nothing is written to a cache."""
    _cuda(rows, bias, positions, seq_of_token, inv_freq)
    _need(rows.stride(1) == 1 and rows.shape[1] >= n_heads * head_dim and head_dim % 2 == 0, "rotate_heads: bad rows")
    if bias is not None:
        _need(bias.dtype == torch.float32 and bias.numel() >= n_heads * head_dim, "rotate_heads: bias must be fp32")
    if inv_freq is not None:
        _need(inv_freq.dtype == torch.float32 and inv_freq.numel() == head_dim // 2, "rotate_heads: inv_freq fp32 [D/2]")
    code = _fn("elementwise", "tw_rope_kv_write")(
        _ptr(rows), c_int(rows.stride(0)), _ptr(None), c_int(0), c_long(0), _ptr(bias), _ptr(positions),
        _ptr(seq_of_token), _ptr(None), _ptr(None),
        c_int(0), _ptr(inv_freq), _ptr(None), _ptr(None), c_int(n_tokens), c_int(n_heads), c_int(0), c_int(head_dim),
        c_int(1), c_int(0), c_int(0), c_int(dtype_code(rows.dtype)), _ptr(None), _stream())
    _check(code, "rotate_heads")


def rotate_pairs(rows: torch.Tensor, positions: torch.Tensor, seq_of_token: torch.Tensor, inv_freq: torch.Tensor,
                 n_tokens: int, n_heads: int, head_dim: int, rot_dims: int, interleaved: bool, magnitude: float = 1.0,
                 first: int = 0) -> None:
    """In place on the first ``n_heads`` heads of each packed row: rotate ``rot_dims / 2`` pairs of every head, from
    the head's value ``first`` on, by ``position * inv_freq[i]``; pair i is (2i, 2i+1) when ``interleaved``, else
    (i, i + rot_dims / 2), counted from ``first``.  cos and sin are both multiplied by ``magnitude``."""
    _cuda(rows, positions, seq_of_token, inv_freq)
    _need(rows.stride(1) == 1 and rows.shape[1] >= n_heads * head_dim, "rotate_pairs: bad rows")
    _need(rot_dims % 2 == 0 and first >= 0 and 0 <= rot_dims <= head_dim - first and inv_freq.dtype == torch.float32
          and inv_freq.numel() == rot_dims // 2, "rotate_pairs: inv_freq must be fp32 [rot_dims / 2], rot_dims even and inside the head")
    code = _fn("elementwise", "tw_rotate_pairs")(_ptr(rows), c_int(rows.stride(0)), _ptr(positions), _ptr(seq_of_token),
                                                 _ptr(inv_freq), c_int(n_tokens), c_int(n_heads), c_int(head_dim), c_int(first),
                                                 c_int(rot_dims), c_int(1 if interleaved else 0), c_float(magnitude),
                                                 c_int(dtype_code(rows.dtype)), _stream())
    _check(code, "rotate_pairs")


def span_rmsnorm(rows: torch.Tensor, n_rows: int, spans: list[tuple[int, int, int, torch.Tensor]], eps: float) -> None:
    """In place: every span ``(first column, heads, head size, weight fp32 [head size])`` of the rows is that many
    heads side by side, each divided by its own root mean square (eps inside the root) and multiplied by the span's
    weight, in fp32.  One or two spans per call."""
    _need(1 <= len(spans) <= 2, "span_rmsnorm: one or two spans")
    _cuda(rows, *(w for _, _, _, w in spans))
    _need(rows.dim() == 2 and rows.stride(1) == 1 and rows.shape[0] >= n_rows, "span_rmsnorm: bad rows")
    for col, heads, dim, w in spans:
        _need(col >= 0 and heads > 0 and dim > 0 and col + heads * dim <= rows.shape[1] and w.dtype == torch.float32
              and w.numel() == dim and w.is_contiguous(), "span_rmsnorm: a span must lie inside the rows, with an fp32 weight per value of a head")
    (c0, h0, d0, w0), (c1, h1, d1, w1) = spans[0], (spans[1] if len(spans) == 2 else (0, 0, 0, None))
    code = _fn("elementwise", "tw_span_rmsnorm")(_ptr(rows), c_int(rows.stride(0)), c_int(n_rows), c_int(len(spans)), c_int(c0),
                                                 c_int(h0), c_int(d0), _ptr(w0), c_int(c1), c_int(h1), c_int(d1), _ptr(w1),
                                                 c_float(eps), c_int(dtype_code(rows.dtype)), _stream())
    _check(code, "span_rmsnorm")


def norm_rotate_store(rows: torch.Tensor, n_tokens: int, spans: list[tuple[int, int, int, torch.Tensor]], eps: float,
                      positions: torch.Tensor, seq_of_token: torch.Tensor, seq_slot: torch.Tensor, block_table: torch.Tensor,
                      k_pages: torch.Tensor, v_pages: torch.Tensor | None, k_col: int, v_col: int, write_cache: bool,
                      status: torch.Tensor, dst0: torch.Tensor | None = None, rot_col: int = 0, rot_dims: int = 0,
                      inv_freq: torch.Tensor | None = None, interleaved: bool = False, magnitude: float = 1.0,
                      gate_col: int = 0, gate_out: torch.Tensor | None = None) -> None:
    """One pass over every token's projected row: the norms of ``spans`` (as ``span_rmsnorm``; span 0 goes to the
    contiguous rows ``dst0`` instead of in place where given), the rotation by position of ``rot_dims`` values from
    column ``rot_col`` on (``rotate_pairs`` on one span), and the store of the key columns (from ``k_col``) and value
    columns (from ``v_col``; ``v_pages`` None: one set of pages) into the token's place in the pages.  ``gate_out``
    (fp32 [rows, heads], or None) receives the sigmoid of as many columns from ``gate_col`` on."""
    _need(len(spans) <= 2, "norm_rotate_store: at most two spans")
    _cuda(rows, positions, seq_of_token, seq_slot, block_table, k_pages, v_pages, status, dst0, inv_freq, gate_out, *(w for _, _, _, w in spans))
    _need(rows.dim() == 2 and rows.stride(1) == 1 and rows.shape[0] >= n_tokens and rows.dtype == k_pages.dtype and k_pages.is_contiguous(),
          "norm_rotate_store: rows of the pages' type, contiguous pages")
    for col, heads, dim, w in spans:
        _need(col >= 0 and heads > 0 and dim > 0 and col + heads * dim <= rows.shape[1] and w.dtype == torch.float32
              and w.numel() == dim and w.is_contiguous(), "norm_rotate_store: a span must lie inside the rows, with an fp32 weight per value of a head")
    _need(dst0 is None or (spans and dst0.is_contiguous() and dst0.dtype == rows.dtype and dst0.shape[0] >= n_tokens
                           and dst0.shape[1] == spans[0][1] * spans[0][2]), "norm_rotate_store: the rows of span 0 must be contiguous and of its width")
    _need(rot_dims % 2 == 0 and rot_dims >= 0 and rot_col >= 0 and rot_col + rot_dims <= rows.shape[1]
          and (rot_dims == 0 or (inv_freq is not None and inv_freq.dtype == torch.float32 and inv_freq.numel() == rot_dims // 2)),
          "norm_rotate_store: the rotated span must lie inside the rows, with an fp32 rate per pair")
    _need(v_pages is None or (v_pages.dtype == rows.dtype and v_pages.is_contiguous() and k_pages.shape[:3] == v_pages.shape[:3]),
          "norm_rotate_store: value pages must be contiguous, of the rows' type and as many as the key pages")
    kv_heads, dk = k_pages.shape[1], k_pages.shape[3]
    dv = 0 if v_pages is None else v_pages.shape[3]
    _need(k_col + kv_heads * dk <= rows.shape[1] and (v_pages is None or v_col + kv_heads * dv <= rows.shape[1]),
          "norm_rotate_store: the key and value columns must lie inside the rows")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "norm_rotate_store: bad block table")
    _need(gate_out is None or (gate_out.dtype == torch.float32 and gate_out.is_contiguous() and gate_out.shape[0] >= n_tokens
                               and 0 <= gate_col and gate_col + gate_out.shape[1] <= rows.shape[1]),
          "norm_rotate_store: the gates must be contiguous fp32 rows, and their columns lie inside the rows")
    (c0, h0, d0, w0) = spans[0] if spans else (0, 0, 0, None)
    (c1, h1, d1, w1) = spans[1] if len(spans) == 2 else (0, 0, 0, None)
    code = _fn("elementwise", "tw_norm_rotate_store")(
        _ptr(rows), c_int(rows.stride(0)), c_int(n_tokens), c_int(len(spans)), c_int(c0), c_int(h0), c_int(d0), _ptr(w0), _ptr(dst0),
        c_int(c1), c_int(h1), c_int(d1), _ptr(w1), c_float(eps), c_int(rot_col), c_int(rot_dims), _ptr(inv_freq),
        c_int(1 if interleaved else 0), c_float(magnitude), c_int(k_col), c_int(v_col), _ptr(positions), _ptr(seq_of_token),
        _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(kv_heads), c_int(dk),
        c_int(dv), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]), c_int(1 if write_cache else 0), c_int(gate_col),
        c_int(0 if gate_out is None else gate_out.shape[1]), _ptr(gate_out), c_int(dtype_code(rows.dtype)), _ptr(status), _stream())
    _check(code, "norm_rotate_store")


def gate_mul(out: torch.Tensor, x: torch.Tensor, gate: torch.Tensor, act: int, n_rows: int) -> None:
    """out = x * act(gate) element by element (``GATE_SIGMOID`` or ``GATE_SILU``), fp32 arithmetic; the three may be
    column slices of wider rows and ``out`` may be ``x``."""
    _cuda(out, x, gate)
    cols = out.shape[1]
    _need(x.shape[1] == cols and gate.shape[1] == cols and out.dtype == x.dtype == gate.dtype
          and out.stride(1) == x.stride(1) == gate.stride(1) == 1 and min(out.shape[0], x.shape[0], gate.shape[0]) >= n_rows,
          "gate_mul: three operands of one type and width")
    _need(act in (GATE_SILU, GATE_SIGMOID), "gate_mul: the activation is silu or sigmoid")
    code = _fn("elementwise", "tw_gate_mul")(_ptr(out), c_int(out.stride(0)), _ptr(x), c_int(x.stride(0)), _ptr(gate),
                                             c_int(gate.stride(0)), c_int(n_rows), c_int(cols), c_int(2 if act == GATE_SILU else 1),
                                             c_int(dtype_code(out.dtype)), _stream())
    _check(code, "gate_mul")


def softcap(logits: torch.Tensor, cap: float | None, scale: float = 1.0) -> None:
    """logits <- scale * logits, then (with a cap) logits <- cap * tanh(logits / cap), in place on contiguous fp32 rows."""
    _cuda(logits)
    _need(logits.dtype == torch.float32 and logits.is_contiguous() and (cap is None or cap > 0), "softcap: contiguous fp32 logits and a positive cap")
    code = _fn("elementwise", "tw_softcap")(_ptr(logits), ctypes.c_longlong(logits.numel()), c_float(scale),
                                            c_float(0.0 if cap is None else cap), _stream())
    _check(code, "softcap")


# what stands between two products of a feed-forward (csrc/common.cuh: tw_activate)
ACT_NONE, ACT_SILU, ACT_GELU_TANH, ACT_RELU_SQUARED = 0, 1, 2, 3
ACTIVATIONS = {"silu": ACT_SILU, "gelu_tanh": ACT_GELU_TANH, "relu_squared": ACT_RELU_SQUARED}


def _bias_check(bias: torch.Tensor | None, n: int, dtype: torch.dtype, what: str) -> None:
    _need(bias is None or (bias.is_cuda and bias.dtype == dtype and bias.dim() == 1 and bias.numel() == n and bias.is_contiguous()),
          f"{what}: the bias must be one contiguous value of the activations' type per output")


def silu_mul(out: torch.Tensor, gate_up, n_rows: int, interleaved: bool = False, act: int = ACT_SILU,
             bias: torch.Tensor | None = None) -> None:
    """out[n, i] = act(gate[n, i]) * up[n, i].  Columns of ``gate_up`` are [all gates | all ups],
    or with ``interleaved`` groups of 16: eight gates followed by their eight ups.  ``gate_up`` may be a
    ``SplitSum`` (fp32 slices of the product, added here in slice order); ``out`` is then bfloat16.  ``bias``
    (in the order of the columns, of the output's type) is added to gates and ups first."""
    inter = out.shape[1]
    _bias_check(bias, 2 * inter, out.dtype, "silu_mul")
    if isinstance(gate_up, SplitSum):
        slices = gate_up.slices
        _cuda(out, slices)
        _need(out.dtype == torch.bfloat16 and out.is_contiguous() and slices.dtype == torch.float32 and slices.dim() == 3
              and slices.shape[1] >= n_rows and slices.shape[2] == 2 * inter and slices[0].is_contiguous()
              and inter % 4 == 0 and (not interleaved or inter % 8 == 0) and out.shape[0] >= n_rows,
              "silu_mul: slices must be fp32 [slices, rows, 2I], the output bf16 [rows, I], I a multiple of 4 (8 interleaved)")
        code = _fn("elementwise", "tw_silu_mul_slices")(_ptr(out), _ptr(slices), c_int(slices.shape[0]), c_long(slices.stride(0)),
                                                        c_int(n_rows), c_int(inter), c_int(1 if interleaved else 0), c_int(act), _ptr(bias),
                                                        _stream())
        _check(code, "silu_mul_slices")
        return
    _cuda(out, gate_up)
    _need(gate_up.shape[1] == 2 * inter and gate_up.is_contiguous() and out.is_contiguous()
          and gate_up.dtype == out.dtype, "silu_mul: gate_up must be contiguous [n, 2I] of the output type")
    _need(not interleaved or inter % 8 == 0, "silu_mul: interleaved columns need a multiple of 8")
    code = _fn("elementwise", "tw_silu_mul")(_ptr(out), _ptr(gate_up), c_int(n_rows), c_int(inter),
                                             c_int(1 if interleaved else 0), c_int(act), _ptr(bias), c_int(dtype_code(out.dtype)),
                                             _stream())
    _check(code, "silu_mul")


def activate_rows(x: torch.Tensor, n_rows: int, act: int, bias: torch.Tensor | None = None) -> None:
    """x[:n_rows] <- act(x[:n_rows] + bias) in place, fp32 arithmetic: a feed-forward without a gate."""
    _cuda(x, bias)
    _need(x.dim() == 2 and x.is_contiguous() and x.shape[0] >= n_rows, "activate_rows: contiguous rows")
    _bias_check(bias, x.shape[1], x.dtype, "activate_rows")
    code = _fn("elementwise", "tw_activate_rows")(_ptr(x), _ptr(bias), c_int(n_rows), c_int(x.shape[1]), c_int(act),
                                                  c_int(dtype_code(x.dtype)), _stream())
    _check(code, "activate_rows")


def attention_generic(out: torch.Tensor, q: torch.Tensor, positions: torch.Tensor, seq_of_token: torch.Tensor,
                      seq_slot: torch.Tensor, block_table: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
                      n_tokens: int, n_q_heads: int, n_kv_heads: int, head_dim: int, window: int, scale: float,
                      status: torch.Tensor, sink: torch.Tensor | None = None,
                      bias_by_distance: torch.Tensor | None = None, gate: torch.Tensor | None = None) -> None:
    """Exact paged causal attention, one block per (token, head).  q may be a column
    slice of the packed qkv buffer (row stride is passed on).  The value pages may have rows of another
    length than the key pages (or be the key pages themselves); the output then has heads of that length.
    ``sink`` fp32 [Hq]: exp(sink[h]) joins the softmax's denominator.  ``bias_by_distance`` fp32 [rows, Hq]: row
    min(position - key position, rows - 1) is added to the scaled score.  ``window``: how far a query sees, as
    ``visible_reach`` makes it.  ``gate`` fp32 [rows, Hq]: each head's output is multiplied by its entry."""
    _cuda(out, q, positions, seq_of_token, seq_slot, block_table, k_pages, v_pages, status, sink, bias_by_distance, gate)
    _gate_check(gate, n_tokens, n_q_heads)
    _need(sink is None or (sink.dtype == torch.float32 and sink.numel() == n_q_heads and sink.is_contiguous()),
          "attention: the sink must be fp32 [Hq]")
    _need(bias_by_distance is None or (bias_by_distance.dtype == torch.float32 and bias_by_distance.dim() == 2
                                       and bias_by_distance.shape[1] == n_q_heads and bias_by_distance.is_contiguous()
                                       and bias_by_distance.shape[0] > 0), "attention: the distance bias must be fp32 [rows, Hq]")
    _need(head_dim <= 1024 and v_pages.shape[3] <= 1024, "attention: head sizes above 1024 are not supported")
    _need(k_pages.shape[3] == head_dim and k_pages.shape[:3] == v_pages.shape[:3] and k_pages.is_contiguous()
          and v_pages.is_contiguous(), "attention: pages must be contiguous [pages, kv_heads, page, head size]")
    _need(n_q_heads % n_kv_heads == 0, "attention: query heads must be a multiple of key/value heads")
    _need(q.stride(1) == 1 and out.stride(1) == 1 and q.dtype == out.dtype == k_pages.dtype, "attention: bad operands")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "attention: bad block table")
    code = _fn("attention_generic", "tw_attn_generic")(
        _ptr(out), c_int(out.stride(0)), _ptr(q), c_int(q.stride(0)), _ptr(positions), _ptr(seq_of_token),
        _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(n_tokens),
        c_int(n_q_heads), c_int(n_kv_heads), c_int(head_dim), c_int(v_pages.shape[3]), c_int(k_pages.shape[2]),
        c_int(k_pages.shape[0]), c_int(window), c_float(scale), _ptr(bias_by_distance),
        c_int(0 if bias_by_distance is None else bias_by_distance.shape[0]), _ptr(sink), _ptr(gate), c_int(dtype_code(q.dtype)),
        _ptr(status), _stream())
    _check(code, "attention_generic")


def visible_reach(window: int | None, chunk: int | None) -> int:
    """How far an attention kernel's queries see, as its ``window`` argument says it (csrc/common.cuh: tw_first_key):
    a sliding window is positive, chunks of positions counted from 0 are negative, 0 is everything."""
    if window and chunk:
        raise ValueError("attention sees a sliding window or its own chunk, not both")
    return int(window) if window else -int(chunk) if chunk else 0


def _gate_check(gate: torch.Tensor | None, n_rows: int, n_q_heads: int) -> None:
    _need(gate is None or (gate.dtype == torch.float32 and gate.dim() == 2 and gate.shape[1] == n_q_heads and gate.shape[0] >= n_rows
                           and gate.is_contiguous()), "attention: the output gate must be fp32 [rows, Hq]")


def attention_prepare(q_out: torch.Tensor, rows, n_tokens: int, n_q_heads: int, n_kv_heads: int, head_dim: int, v_dim: int,
                      positions: torch.Tensor, seq_of_token: torch.Tensor, seq_slot: torch.Tensor, block_table: torch.Tensor,
                      k_pages: torch.Tensor, v_pages: torch.Tensor, write_cache: bool, status: torch.Tensor, rot_dims: int = 0,
                      inv_freq: torch.Tensor | None = None, interleaved: bool = False, magnitude: float = 1.0,
                      gate: torch.Tensor | None = None, leave_values: torch.Tensor | None = None,
                      mix_values: torch.Tensor | None = None, mix_weight: torch.Tensor | None = None) -> None:
    """One pass over every token's projected row ``[q heads | k heads | v heads | one number per q head, with gate]``
    (a tensor of the pages' type, or a ``SplitSum``): rotate the first ``rot_dims`` values of every q and k head by
    position, write q to ``q_out`` [rows, Hq D], k and v to the token's place in the pages, and the sigmoid of the last
    columns to ``gate`` (fp32 [rows, Hq]).  ``leave_values`` [rows, Hkv Dv] also receives the values; ``mix_values``
    (what another layer left that way) is blended in before they are stored: (1 - w) v + w mix, w = ``mix_weight`` (an
    fp32 tensor of one number)."""
    _cuda(q_out, positions, seq_of_token, seq_slot, block_table, k_pages, v_pages, status, inv_freq, gate, leave_values, mix_values, mix_weight)
    need = n_q_heads * head_dim + n_kv_heads * (head_dim + v_dim) + (n_q_heads if gate is not None else 0)
    partial, nsplit, split_stride, stride = None, 0, 0, 0
    if isinstance(rows, SplitSum):
        partial, rows = rows.slices, None
        nsplit, split_stride, width = partial.shape[0], partial.stride(0), partial.shape[2]
        _need(partial.is_cuda and partial.dtype == torch.float32 and partial[0].is_contiguous() and partial.shape[1] >= n_tokens,
              "attention_prepare: bad split source")
    else:
        _cuda(rows)
        width, stride = rows.shape[1], rows.stride(0)
        _need(rows.dtype == k_pages.dtype and rows.stride(1) == 1 and rows.shape[0] >= n_tokens, "attention_prepare: bad rows")
    _need(width >= need, f"attention_prepare: a row has {width} columns, {need} are needed")
    _need(q_out.dtype == k_pages.dtype == v_pages.dtype and q_out.is_contiguous() and q_out.shape[0] >= n_tokens
          and q_out.shape[1] == n_q_heads * head_dim, "attention_prepare: q must be contiguous [rows, Hq D] of the pages' type")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and tuple(k_pages.shape[1:]) == (n_kv_heads, k_pages.shape[2], head_dim)
          and tuple(v_pages.shape) == (*k_pages.shape[:3], v_dim), "attention_prepare: pages must be contiguous [pages, kv_heads, page, head size]")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "attention_prepare: bad block table")
    _need(rot_dims % 2 == 0 and 0 <= rot_dims <= head_dim and (rot_dims == 0 or (
        inv_freq is not None and inv_freq.dtype == torch.float32 and inv_freq.numel() == rot_dims // 2)), "attention_prepare: one fp32 rate per pair")
    _gate_check(gate, n_tokens, n_q_heads)
    _need(leave_values is None or mix_values is None, "attention_prepare: values are left or mixed, not both")
    first = leave_values if leave_values is not None else mix_values
    _need(first is None or (first.dtype == q_out.dtype and first.is_contiguous() and first.shape[0] >= n_tokens
                            and first.shape[1] == n_kv_heads * v_dim), "attention_prepare: the kept values must be contiguous [rows, Hkv Dv]")
    _need(mix_values is None or (mix_weight is not None and mix_weight.dtype == torch.float32 and mix_weight.numel() == 1),
          "attention_prepare: mixing needs an fp32 weight")
    role = 1 if leave_values is not None else 2 if mix_values is not None else 0
    code = _fn("attention_prepare", "tw_attention_prepare")(
        _ptr(q_out), _ptr(rows), c_int(stride), _ptr(partial), c_int(nsplit), c_long(split_stride), c_int(width), c_int(n_tokens),
        c_int(n_q_heads), c_int(n_kv_heads), c_int(head_dim), c_int(v_dim), c_int(rot_dims), c_int(1 if interleaved else 0),
        c_float(magnitude), _ptr(inv_freq), c_int(role), _ptr(mix_weight), _ptr(first), _ptr(gate), _ptr(positions), _ptr(seq_of_token),
        _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(k_pages.shape[2]),
        c_int(k_pages.shape[0]), c_int(1 if write_cache else 0), c_int(dtype_code(q_out.dtype)), _ptr(status), _stream())
    _check(code, "attention_prepare")


def sample(out: torch.Tensor, logits: torch.Tensor, n_rows: int, temperature: torch.Tensor | None = None,
           seed: torch.Tensor | None = None, counter: torch.Tensor | None = None) -> None:
    """out[r] = chosen token of row r (int32).  Rows with temperature 0 are greedy."""
    _cuda(out, logits, temperature, seed, counter)
    _need(logits.dtype == torch.float32 and logits.is_contiguous() and logits.dim() == 2, "sample: logits fp32 [rows, vocab]")
    _need(out.dtype == torch.int32 and out.numel() >= n_rows, "sample: out must be int32")
    if temperature is not None:
        _need(temperature.dtype == torch.float32 and seed is not None and counter is not None
              and seed.dtype == torch.int64 and counter.dtype == torch.int64, "sample: temperature fp32, seed/counter int64")
    code = _fn("sampling", "tw_sample")(_ptr(out), _ptr(logits), c_int(n_rows), c_int(logits.shape[1]),
                                        _ptr(temperature), _ptr(seed), _ptr(counter), _stream())
    _check(code, "sample")


# ---------------------------------------------------------------------------
# bf16 tensor-core attention (one compiled library per head size)
# ---------------------------------------------------------------------------
DECODE_MAX_SPLITS = 128          # most slices of a request's keys (the merge keeps two floats per head and slice in shared memory)
DECODE_SCRATCH_UNITS = 1024      # most (request, split) pairs whose partial results fit the scratch buffer
_SM_COUNT = 148


def tensor_core_attention_supported(dtype: torch.dtype, head_dim: int, v_dim: int | None = None) -> bool:
    """``v_dim``: the size of a value where it differs from ``head_dim``."""
    return dtype == torch.bfloat16 and all(d % 16 == 0 and 16 <= d <= 256 for d in (head_dim, v_dim or head_dim))


def head_size_defines(head_dim: int, v_dim: int) -> dict[str, int]:
    """The compile-time sizes an attention library is built for."""
    return {"TW_HEAD_DIM": head_dim} if v_dim == head_dim else {"TW_HEAD_DIM": head_dim, "TW_V_DIM": v_dim}


def tcgen05_attention_supported(dtype: torch.dtype, head_dim: int, page_size: int, v_dim: int | None = None) -> bool:
    """The tcgen05 prefill attention takes bfloat16, head sizes 64 and 128, values of 32, 64 or 128, and pages of at least
    8 keys that divide a tile of 128 keys or are a multiple of it."""
    return (dtype == torch.bfloat16 and head_dim in (64, 128) and (v_dim or head_dim) in (32, 64, 128) and page_size >= 8
            and (128 % page_size == 0 or page_size % 128 == 0))


TCGEN05_ATTENTION_MIN_TOKENS = 128


def prefer_tcgen05_attention(dtype: torch.dtype, head_dim: int, page_size: int, max_q_len: int, v_dim: int | None = None) -> bool:
    """Whether a step whose longest portion has ``max_q_len`` tokens runs its prompt attention on
    the tcgen05 kernel.  TESSWEAVE_PREFILL_ATTENTION=mma|tcgen05 forces one of the two (the latter
    only for shapes the kernel takes)."""
    import os
    if not tcgen05_attention_supported(dtype, head_dim, page_size, v_dim):
        return False
    forced = os.environ.get("TESSWEAVE_PREFILL_ATTENTION")
    if forced == "mma":
        return False
    if forced == "tcgen05":
        return True
    return max_q_len >= TCGEN05_ATTENTION_MIN_TOKENS


def decode_blocks_per_sm(v_dim: int) -> int:
    """How many blocks of the split-KV kernel that loads keys through registers an SM holds: four, or as many as the
    shared memory of their value stages (three stages of 64 padded rows) leaves room for."""
    return max(1, min(4, 227 * 1024 // (3 * 64 * (v_dim + 8) * 2 + 4096)))


def decode_splits(n_seqs: int, n_kv_heads: int, group: int, max_kv_len: int, v_dim: int = 128) -> int:
    """How many slices the keys of a request are cut into, so that the launch fills the GPU.
    Up to 16 slices merge inside a thread-block cluster, which saves 2-3 us over the merge through
    scratch memory; clusters of 15 and 16 are only placed well when there are few of them, so with many
    (request, head) groups 15 and 16 slices become 14 (measured on B200, batch 8, 4 key/value heads,
    4096 keys, a whole decode step: 3.61 ms with 13 or 14 slices, 3.64 with 12, 3.94 with 16, 4.02 with 15).
    Values of more than 128 leave fewer blocks on an SM, and a launch of more blocks than fit at once pays for every
    further one (28 heads over cached rows of 256 values, batch 8, 4,096 keys, the kernel alone: 29.6 us with 8 slices on
    256 blocks, 46 to 62 with 9 to 16)."""
    import os
    forced = os.environ.get("TESSWEAVE_DECODE_SPLITS")
    if forced:
        return max(1, min(int(forced), 128, DECODE_SCRATCH_UNITS // max(1, n_seqs)))
    head_tiles = (group + 7) // 8
    tiles = max(1, -(-max_kv_len // 64))
    groups = max(1, n_seqs * n_kv_heads * head_tiles)
    # the kernel fits four blocks on an SM (fewer with wide values); aim at a little under one full wave of blocks
    fits = decode_blocks_per_sm(v_dim)
    room, full = 7 * fits * _SM_COUNT // 8, 15 * fits * _SM_COUNT // 16
    target = max(1, (room + groups // 2) // groups)        # rounded: 1.9 blocks' worth of room is two slices
    if target > 4 and target * groups > room:
        # clusters of five and more blocks are no longer all placed at once when the launch has more than 3.5 blocks
        # per SM (batch 12, 4 key/value heads, a whole decode step: 3.81 ms with 10 slices, 4.21 with 11)
        target = max(4, room // groups)
    elif 1 < target <= 4 and target * groups > full:
        # small clusters fill the SMs a little further (batch 44: 528 blocks of 3 slices, 5.23 ms against 5.51 with 2),
        # but not to the last slot (batch 48: 576 blocks, 6.56 ms against 5.59 with 2)
        target = max(1, full // groups)
    nsplit = max(1, min(tiles, target, 128, DECODE_SCRATCH_UNITS // max(1, n_seqs)))
    if 16 < nsplit <= 64 and max_kv_len <= 8192:
        # up to 8,192 keys the merge inside a cluster beats more slices merged through scratch memory (4,096 keys:
        # batch 3 / 4 / 6 steps take 3.24 / 3.26 / 3.37 ms with 14-16 slices against 3.30 / 3.33 / 3.52 with 21-32);
        # with longer contexts and few requests more slices win (16,384 keys, batch 2: 3.62 ms with 64, 3.83 with 16)
        nsplit = 16
    if 14 < nsplit <= 16 and groups > 8:
        nsplit = 14          # at every context length: 16,384 keys 4.53 ms with 14 slices, 5.20 with 16; 32,768 keys 5.85 and 7.05
    # the kernel cuts the keys into slices of a multiple of 64 keys: no slice without keys
    per = -(-(-(-max_kv_len // nsplit)) // 64) * 64
    return max(1, -(-max_kv_len // per))


def decode_scratch_floats(n_q_heads: int, head_dim: int) -> int:
    return DECODE_SCRATCH_UNITS * n_q_heads * (head_dim + 2)


def decode_counter_ints(n_seqs: int, n_kv_heads: int, group: int) -> int:
    """int32 counters (zero before the first launch, left zero by every launch) the split
    decode kernel uses to find the block that finishes last."""
    return max(n_seqs, DECODE_SCRATCH_UNITS) * n_kv_heads * ((group + 7) // 8)


def _attn_common_checks(out, q, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim):
    _need(tensor_core_attention_supported(q.dtype, head_dim, v_pages.shape[3]),
          f"tensor-core attention takes bfloat16 and head sizes that are multiples of 16 up to 256, not {q.dtype}/{head_dim}/{v_pages.shape[3]}")
    _need(n_q_heads % n_kv_heads == 0, "attention: query heads must be a multiple of key/value heads")
    _need(q.stride(1) == 1 and out.stride(1) == 1 and out.dtype == q.dtype == k_pages.dtype == v_pages.dtype,
          "attention: operands must be bfloat16 with unit inner stride")
    _need(q.stride(0) % 2 == 0 and q.storage_offset() % 2 == 0 and out.stride(0) % 2 == 0, "attention: rows must be 4-byte aligned")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.shape[3] == head_dim
          and k_pages.shape[1] == n_kv_heads and k_pages.shape[:3] == v_pages.shape[:3],
          "attention: cache pages must be contiguous [pages, kv_heads, page, head_dim]")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "attention: bad block table")


def _score_terms_checks(sink, bias_rows, n_q_heads):
    _need(sink is None or (sink.dtype == torch.float32 and sink.numel() == n_q_heads and sink.is_contiguous()),
          "attention: the sink must be fp32 [Hq]")
    _need(bias_rows is None or (bias_rows.dtype == torch.float32 and bias_rows.dim() == 2 and bias_rows.shape[0] == n_q_heads
                                and bias_rows.shape[1] > 0 and bias_rows.is_contiguous()),
          "attention: the distance bias of the tensor-core kernels must be fp32 [Hq, distances]")


def attention_decode(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, n_seqs,
                     n_q_heads, n_kv_heads, head_dim, window, scale, nsplit, scratch, counters, status,
                     merge_in_scratch: bool = False, sink: torch.Tensor | None = None,
                     bias_rows: torch.Tensor | None = None, gate: torch.Tensor | None = None) -> None:
    """Split-KV attention for the requests of the batch that bring one token (others are skipped).
    Up to 16 slices merge inside a thread-block cluster; more (or all, with ``merge_in_scratch``)
    merge through ``scratch`` (fp32, the slices' partial results) and ``counters`` (int32, all
    zero, left zero), which find the block that finishes last.  ``sink`` fp32 [Hq]: exp(sink[h]) joins the
    denominator of head h.  ``bias_rows`` fp32 [Hq, distances]: entry min(position - key position, distances - 1)
    of head h is added to its scaled score.  ``v_pages`` may be ``k_pages`` (values that are the keys).
    ``window``: how far a query sees, as ``visible_reach`` makes it.  ``gate`` fp32 [rows, Hq]: each head's output of a
    row is multiplied by its entry.  The value pages may have rows of another length; the output has heads of that length."""
    _cuda(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, scratch, counters, status,
          sink, bias_rows, gate)
    _gate_check(gate, 0, n_q_heads)
    v_dim = v_pages.shape[3]
    _attn_common_checks(out, q, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim)
    _score_terms_checks(sink, bias_rows, n_q_heads)
    _need(out.stride(0) % 4 == 0 and out.data_ptr() % 8 == 0, "attention_decode: output rows must be 8-byte aligned")
    _need(q.data_ptr() % 16 == 0 and q.stride(0) % 8 == 0, "attention_decode: rows of q must be 16-byte aligned")
    _need(1 <= nsplit <= DECODE_MAX_SPLITS, f"attention_decode: 1 to {DECODE_MAX_SPLITS} slices, not {nsplit}")
    if nsplit > 1:
        _need(scratch is not None and scratch.dtype == torch.float32 and scratch.data_ptr() % 16 == 0
              and scratch.numel() >= n_seqs * n_q_heads * nsplit * (v_dim + 2), "attention_decode: scratch too small")
        _need(counters is not None and counters.dtype == torch.int32
              and counters.numel() >= n_seqs * n_kv_heads * ((n_q_heads // n_kv_heads + 7) // 8),
              "attention_decode: too few counters")
    head = (_ptr(out), c_int(out.stride(0)), _ptr(q), c_int(q.stride(0)), _ptr(seq_q_start), _ptr(seq_q_len),
            _ptr(seq_kv_len), _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages),
            c_int(n_seqs), c_int(n_q_heads), c_int(n_kv_heads), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]),
            c_int(window), c_float(scale), c_int(nsplit), c_int(1 if merge_in_scratch else 0), _ptr(scratch), _ptr(counters))
    defines = head_size_defines(head_dim, v_dim)
    if sink is None and bias_rows is None and gate is None:
        code = _fn("attention_bf16", "tw_attn_decode", defines)(*head, _ptr(status), _stream())
    else:
        code = _fn("attention_bf16", "tw_attn_decode_terms", defines)(
            *head, _ptr(bias_rows), c_int(0 if bias_rows is None else bias_rows.shape[1]), _ptr(sink), _ptr(gate), _ptr(status), _stream())
    _check(code, "attention_decode")


WEIGHT_PREFETCH_BYTES = 24 << 20


def weight_prefetch_bytes() -> int:
    """How much of the weights that the part after the attention streams first (the feed-forward's first matrix)
    a decode step's attention asks into L2 while its slices merge.  Measured on a 7B-size layer: 24 to 32 MB is
    best at 1, 8 and 64 requests; more competes with the output product that runs in between, and asking for
    that product's own matrix gains nothing.  TESSWEAVE_WEIGHT_PREFETCH_MB overrides it; 0 switches it off."""
    import os
    mb = os.environ.get("TESSWEAVE_WEIGHT_PREFETCH_MB")
    return WEIGHT_PREFETCH_BYTES if mb is None else max(0, int(mb)) << 20


PRODUCT_PREFETCH_BYTES = 16 << 20


def weight_head(w: torch.Tensor | None, nbytes: int, skip_bytes: int = 0) -> torch.Tensor | None:
    """``nbytes`` of a contiguous weight from byte ``skip_bytes`` on as a flat view (what there is of them), or None."""
    if w is None or nbytes <= 0 or not w.is_contiguous():
        return None
    size = w.element_size()
    part = w.view(-1)[skip_bytes // size: (skip_bytes + nbytes) // size]
    return part if part.numel() else None


OUTPUT_PRODUCT_PREFETCH_BYTES = 24 << 20


def output_product_prefetch_bytes() -> int:
    """How much more of the feed-forward's first matrix the attention's output product asks into L2 when its own
    stream of weights ends, after what the attention kernel asked for.  The feed-forward's product is resident by
    then and fetches its first rows itself; these are rows it reaches later.  Measured on a 7B-size layer, whole
    decode steps: 8 / 16 / 24 / 32 / 48 / 64 / 96 MB give 0.6 / 1.0 / 1.2 / 1.2 / 1.1 / 0.6 / 0 % at 8 requests and
    the same at one; at the 14B sizes 16 and 24 MB are better than 32 (one request: 2 and 1 %).
    TESSWEAVE_OUTPUT_PREFETCH_MB overrides it; 0 switches it off."""
    import os
    mb = os.environ.get("TESSWEAVE_OUTPUT_PREFETCH_MB")
    return OUTPUT_PRODUCT_PREFETCH_BYTES if mb is None else max(0, int(mb)) << 20


def product_prefetch_bytes() -> int:
    """How much of the next matrix a small-batch product asks into L2 when its own stream of weights ends
    (gate/up before down).  Measured on a 7B-size layer: 8 to 24 MB are alike, 0.6 to 0.8 % of a step at 1 and 8
    requests.  Before a product that is resident early (q/k/v behind the norm, the attention's output product)
    the same request makes the step slower, so only the feed-forward uses it.  TESSWEAVE_PRODUCT_PREFETCH_MB
    overrides it; 0 switches it off."""
    import os
    mb = os.environ.get("TESSWEAVE_PRODUCT_PREFETCH_MB")
    return PRODUCT_PREFETCH_BYTES if mb is None else max(0, int(mb)) << 20


def weight_prefetch_min_cache_bytes() -> int:
    """The attention of a decode step prefetches weights only if it reads at least this much of the cache: a
    shorter kernel ends while the output product still fetches its own matrix, and the prefetch gets in its way
    (one request at 512 keys of a 7B-size layer: 1.4% slower with it).  TESSWEAVE_WEIGHT_PREFETCH_MIN_KB overrides."""
    import os
    kb = os.environ.get("TESSWEAVE_WEIGHT_PREFETCH_MIN_KB")
    return (2 << 20) if kb is None else int(kb) << 10


def fused_decode_enabled() -> bool:
    """TESSWEAVE_FUSED_DECODE=0 keeps bias, rotation and cache write of decode-only steps in a kernel of their own."""
    import os
    return os.environ.get("TESSWEAVE_FUSED_DECODE", "1") != "0"


def attention_decode_fused(out, source, bias, inv_freq, write_cache, seq_q_start, seq_q_len, seq_kv_len, seq_slot,
                           block_table, k_pages, v_pages, n_seqs, n_q_heads, n_kv_heads, head_dim, window, scale,
                           nsplit, scratch, counters, status, merge_in_scratch: bool = False,
                           prefetch: torch.Tensor | None = None) -> None:
    """Decode attention straight from the q/k/v product of a decode-only step: the kernel adds ``bias``,
    rotates q and k by position (``inv_freq``), writes the new key and value into their cache pages
    (``write_cache``) and attends.  ``source`` is the product: a ``SplitSum`` of fp32 slices or a bf16
    [rows, (Hq + 2 Hkv) D] tensor.  ``prefetch``: a contiguous tensor the next kernel streams (its weights);
    the blocks ask for it to be brought into L2 once their keys are in.  The other arguments are those of
    ``attention_decode``."""
    width = (n_q_heads + 2 * n_kv_heads) * head_dim
    partial = dense = None
    nslices = slice_stride = dense_stride = 0
    if isinstance(source, SplitSum):
        partial = source.slices
        _need(partial.is_cuda and partial.dtype == torch.float32 and partial.dim() == 3 and partial.shape[2] == width
              and partial[0].is_contiguous(), "attention_decode_fused: bad split source")
        nslices, slice_stride = partial.shape[0], partial.stride(0)
    else:
        dense = source
        _need(dense.is_cuda and dense.dtype == torch.bfloat16 and dense.dim() == 2 and dense.shape[1] == width
              and dense.stride(1) == 1, "attention_decode_fused: the product must be bf16 [rows, (Hq + 2 Hkv) D]")
        dense_stride = dense.stride(0)
    _cuda(out, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, scratch, counters, status,
          bias, inv_freq)
    _need(tensor_core_attention_supported(out.dtype, head_dim) and out.dtype == k_pages.dtype == v_pages.dtype,
          "attention_decode_fused: bfloat16 and a head size that is a multiple of 16 up to 256")
    _need(n_q_heads % n_kv_heads == 0, "attention: query heads must be a multiple of key/value heads")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.shape[3] == head_dim
          and k_pages.shape[1] == n_kv_heads and v_pages.shape == k_pages.shape,
          "attention: cache pages must be contiguous [pages, kv_heads, page, head_dim]")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "attention: bad block table")
    _need(out.stride(1) == 1 and out.stride(0) % 4 == 0 and out.data_ptr() % 8 == 0,
          "attention_decode_fused: output rows must be 8-byte aligned")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == width), "attention_decode_fused: bias must be fp32")
    _need(inv_freq is None or (inv_freq.dtype == torch.float32 and inv_freq.numel() == head_dim // 2),
          "attention_decode_fused: inv_freq must be fp32 [D/2]")
    _need(1 <= nsplit <= DECODE_MAX_SPLITS, f"attention_decode_fused: 1 to {DECODE_MAX_SPLITS} slices, not {nsplit}")
    if nsplit > 1:
        _need(scratch is not None and scratch.dtype == torch.float32 and scratch.data_ptr() % 16 == 0
              and scratch.numel() >= n_seqs * n_q_heads * nsplit * (head_dim + 2), "attention_decode: scratch too small")
        _need(counters is not None and counters.dtype == torch.int32
              and counters.numel() >= n_seqs * n_kv_heads * ((n_q_heads // n_kv_heads + 7) // 8),
              "attention_decode: too few counters")
    code = _fn("attention_bf16", "tw_attn_decode_fused", {"TW_HEAD_DIM": head_dim})(
        _ptr(out), c_int(out.stride(0)), _ptr(partial), c_int(nslices), ctypes.c_longlong(slice_stride), _ptr(dense),
        c_int(dense_stride), _ptr(bias), _ptr(inv_freq), c_int(1 if write_cache else 0), _ptr(seq_q_start), _ptr(seq_q_len),
        _ptr(seq_kv_len), _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages),
        c_int(n_seqs), c_int(n_q_heads), c_int(n_kv_heads), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]),
        c_int(window), c_float(scale), c_int(nsplit), c_int(1 if merge_in_scratch else 0), _ptr(scratch), _ptr(counters),
        _ptr(status), _ptr(prefetch), ctypes.c_longlong(prefetch.numel() * prefetch.element_size() if prefetch is not None else 0),
        _stream())
    _check(code, "attention_decode_fused")


# ---------------------------------------------------------------------------
# decode attention fed by TMA (head sizes that are multiples of 64)
# ---------------------------------------------------------------------------
def decode_tma_supported(dtype: torch.dtype, head_dim: int, page_size: int, v_dim: int | None = None) -> bool:
    """Whether single-token requests attend through ``attention_decode_tma``: bfloat16, a head size of 64, 128,
    192 or 256, and pages that are a whole fraction (at least 4 keys) or a whole multiple of a 64-key tile.
    TESSWEAVE_DECODE_TMA=0 keeps the kernel that loads keys through registers."""
    import os
    if os.environ.get("TESSWEAVE_DECODE_TMA", "1") == "0":
        return False
    return (dtype == torch.bfloat16 and all(d % 64 == 0 and 64 <= d <= 256 for d in (head_dim, v_dim or head_dim)) and page_size >= 4
            and (64 % page_size == 0 or page_size % 64 == 0))


def decode_tma_splits(n_seqs: int, n_kv_heads: int, group: int, max_kv_len: int) -> int:
    """How many slices the TMA decode attention cuts a request's keys into.  Two blocks share an SM (a ring of
    three 64-key tiles each), and a block alone does not pull its share of the bandwidth, so the launch is filled
    to about 256 blocks -- not to the last of the 296 places: clusters that do not all find room at once start a
    second round (measured on B200 at 4,096 keys, whole decode steps of the 7B-sized model: batch 8 with 8 slices
    3.33 ms, with 4 slices 3.53, with 9 (288 blocks) 3.75; batch 12 with 5 slices 3.61 ms, with 6 (288 blocks)
    4.07, with 3 (144 blocks) 4.71; batch 4 with 13 slices 3.15 ms, with 14 or 16 3.5; batch 2 with 8 slices 3.18
    ms, with 12 or 16 3.4 to 3.5).  Few requests with long contexts take more slices and merge through scratch
    memory (16,384 keys, batch 2, 12 layers: 1.56 ms with 32 slices, 1.89 with 16).
    TESSWEAVE_DECODE_SPLITS forces a number."""
    import os
    forced = os.environ.get("TESSWEAVE_DECODE_SPLITS")
    tiles = max(1, -(-max_kv_len // 64))
    most = min(tiles, DECODE_MAX_SPLITS, DECODE_SCRATCH_UNITS // max(1, n_seqs))
    if forced:
        return max(1, min(int(forced), most))
    groups = max(1, n_seqs * n_kv_heads * ((group + 7) // 8))
    if groups <= 8 and max_kv_len > 8192:
        want = min(32, 256 // groups)
    elif groups <= 4:
        want = 16
    elif groups <= 8:
        want = 8
    elif groups <= 16:
        want = 13
    else:
        want = max(1, 256 // groups)
    nsplit = max(1, min(want, most))
    per = -(-(-(-max_kv_len // nsplit)) // 64) * 64          # slices are whole tiles: no slice without keys
    return max(1, -(-max_kv_len // per))


DECODE_TMA_CLUSTER_SLICES = 16      # more slices than this merge through scratch memory, without clusters


def decode_attention_resident_early(blocks: int, nsplit: int) -> bool:
    """Whether the q/k/v product of a decode-only step lets the TMA decode attention become resident while it runs
    (griddepcontrol.launch_dependents at its start), so that the attention's copies are under way when the
    product ends.  Clusters are only all placed at once on a GPU that is mostly free: measured on B200, whole
    steps of the 7B-sized model, with the trigger against without: 40 to 64 blocks (1 or 2 requests) 1.4 to 1.7 %
    faster, 144 and 156 blocks (4 requests at 512 keys, 3 at 4,096) 1.7 and 1.1 % faster, 208 blocks (4 requests
    at 4,096 keys) 9 % slower, 256 blocks (8 requests) 5 to 10 % slower; launches that merge through scratch
    memory (no clusters) 1 % faster at 128 and at 256 blocks.  TESSWEAVE_DECODE_EARLY=0/1 forces it."""
    import os
    forced = os.environ.get("TESSWEAVE_DECODE_EARLY")
    if forced is not None:
        return forced == "1"
    return nsplit > DECODE_TMA_CLUSTER_SLICES or blocks * 10 <= _SM_COUNT * 11


def attention_decode_tma(out, q, source, bias, inv_freq, write_cache, seq_q_start, seq_q_len, seq_kv_len, seq_slot,
                         block_table, k_pages, v_pages, n_seqs, n_q_heads, n_kv_heads, head_dim, window, scale, nsplit,
                         scratch, counters, status, merge_in_scratch: bool = False, prefetch: torch.Tensor | None = None,
                         stages: int = 0, gate: torch.Tensor | None = None) -> None:
    """Split-KV attention for the requests of the batch that bring one token, keys and values brought in by TMA.
    Either ``q`` (bf16 [rows, Hq D], 16-byte aligned rows) or ``source`` -- the step's untouched q/k/v product, a
    ``SplitSum`` or a bf16 [rows, (Hq + 2 Hkv) D] tensor, which the kernel biases, rotates and (``write_cache``)
    stores itself -- is given.  The other arguments are those of ``attention_decode`` / ``attention_decode_fused``;
    ``stages`` is the depth of a block's ring of 64-key tiles (0: chosen from the size of the launch).  ``window`` and
    ``gate``: as for ``attention_decode``; with ``q`` the values may have another size than the keys."""
    import os
    width = (n_q_heads + 2 * n_kv_heads) * head_dim
    partial = dense = None
    nslices = slice_stride = dense_stride = 0
    if isinstance(source, SplitSum):
        partial = source.slices
        _need(partial.is_cuda and partial.dtype == torch.float32 and partial.dim() == 3 and partial.shape[2] == width
              and partial[0].is_contiguous(), "attention_decode_tma: bad split source")
        nslices, slice_stride = partial.shape[0], partial.stride(0)
    elif source is not None:
        dense = source
        _need(dense.is_cuda and dense.dtype == torch.bfloat16 and dense.dim() == 2 and dense.shape[1] == width
              and dense.stride(1) == 1, "attention_decode_tma: the product must be bf16 [rows, (Hq + 2 Hkv) D]")
        dense_stride = dense.stride(0)
    else:
        _need(q is not None and q.is_cuda and q.dtype == torch.bfloat16 and q.stride(1) == 1 and q.data_ptr() % 16 == 0
              and q.stride(0) % 8 == 0, "attention_decode_tma: q must be bf16 with 16-byte aligned rows")
    _cuda(out, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, scratch, counters, status,
          bias, inv_freq, prefetch, gate)
    _gate_check(gate, 0, n_q_heads)
    v_dim = v_pages.shape[3]
    _need(decode_tma_supported(out.dtype, head_dim, k_pages.shape[2], v_dim) or os.environ.get("TESSWEAVE_DECODE_TMA") == "0",
          f"attention_decode_tma does not take head size {head_dim} with pages of {k_pages.shape[2]} keys in {out.dtype}")
    _need(out.dtype == k_pages.dtype == v_pages.dtype == torch.bfloat16, "attention_decode_tma: bfloat16 only")
    _need(n_q_heads % n_kv_heads == 0, "attention: query heads must be a multiple of key/value heads")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.shape[3] == head_dim
          and k_pages.shape[1] == n_kv_heads and v_pages.shape[:3] == k_pages.shape[:3] and (source is None or v_dim == head_dim)
          and k_pages.data_ptr() % 16 == 0 and v_pages.data_ptr() % 16 == 0,
          "attention: cache pages must be contiguous, 16-byte aligned [pages, kv_heads, page, head_dim]")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "attention: bad block table")
    _need(out.stride(1) == 1 and out.stride(0) % 4 == 0 and out.data_ptr() % 8 == 0,
          "attention_decode_tma: output rows must be 8-byte aligned")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == width), "attention_decode_tma: bias must be fp32")
    _need(inv_freq is None or (inv_freq.dtype == torch.float32 and inv_freq.numel() == head_dim // 2),
          "attention_decode_tma: inv_freq must be fp32 [D/2]")
    _need(1 <= nsplit <= DECODE_MAX_SPLITS, f"attention_decode_tma: 1 to {DECODE_MAX_SPLITS} slices, not {nsplit}")
    if nsplit > 1:
        _need(scratch is not None and scratch.dtype == torch.float32 and scratch.data_ptr() % 16 == 0
              and scratch.numel() >= n_seqs * n_q_heads * nsplit * (v_dim + 2), "attention_decode: scratch too small")
        _need(counters is not None and counters.dtype == torch.int32
              and counters.numel() >= n_seqs * n_kv_heads * ((n_q_heads // n_kv_heads + 7) // 8),
              "attention_decode: too few counters")
    stages = stages or int(os.environ.get("TESSWEAVE_DECODE_STAGES", "0"))
    code = _fn("attention_decode_tma", "tw_attn_decode_tma", head_size_defines(head_dim, v_dim))(
        _ptr(out), c_int(out.stride(0)), _ptr(q), c_int(q.stride(0) if q is not None else 0), _ptr(partial), c_int(nslices),
        ctypes.c_longlong(slice_stride), _ptr(dense), c_int(dense_stride), _ptr(bias), _ptr(inv_freq),
        c_int(1 if write_cache else 0), _ptr(seq_q_start), _ptr(seq_q_len), _ptr(seq_kv_len), _ptr(seq_slot),
        _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(n_seqs), c_int(n_q_heads),
        c_int(n_kv_heads), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]), c_int(window), c_float(scale), c_int(nsplit),
        c_int(stages), c_int(1 if merge_in_scratch else 0), _ptr(scratch), _ptr(counters), _ptr(status), _ptr(prefetch),
        ctypes.c_longlong(prefetch.numel() * prefetch.element_size() if prefetch is not None else 0), _ptr(gate), _stream())
    _check(code, "attention_decode_tma")


def attention_prefill_tcgen05(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, n_seqs,
                              max_q_len, n_q_heads, n_kv_heads, head_dim, window, scale, skip_single, status,
                              gate: torch.Tensor | None = None) -> None:
    """The same as ``attention_prefill`` on the 5th-generation tensor cores (TMA, tcgen05.mma,
    accumulators in tensor memory), for the shapes ``tcgen05_attention_supported`` names and a positive scale."""
    _cuda(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, status, gate)
    _gate_check(gate, 0, n_q_heads)
    _attn_common_checks(out, q, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim)
    _need(tcgen05_attention_supported(q.dtype, head_dim, k_pages.shape[2], v_pages.shape[3]),
          f"tcgen05 attention does not take head size {head_dim} with pages of {k_pages.shape[2]} keys")
    _need(q.stride(0) % 8 == 0 and out.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0 and out.data_ptr() % 16 == 0,
          "tcgen05 attention: rows of q and out must be 16-byte aligned")
    code = _fn("attention_tcgen05", "tw_attn_prefill_tc5", head_size_defines(head_dim, v_pages.shape[3]))(
        _ptr(out), c_int(out.stride(0)), _ptr(q), c_int(q.stride(0)), _ptr(seq_q_start), _ptr(seq_q_len),
        _ptr(seq_kv_len), _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages),
        c_int(n_seqs), c_int(max_q_len), c_int(n_q_heads), c_int(n_kv_heads), c_int(k_pages.shape[2]),
        c_int(k_pages.shape[0]), c_int(window), c_float(scale), c_int(1 if skip_single else 0), _ptr(gate), _ptr(status), _stream())
    _check(code, "attention_prefill_tcgen05")


LATENT_TCGEN05_MIN_KEYS = 256


def latent_tcgen05_key_tile(page_size: int) -> int | None:
    """Keys per tile of the latent tcgen05 attention for pages of this size, or None: a tile is a whole number of pages (at
    most 32), or a page a whole number of tiles."""
    if page_size >= 4 and 96 % page_size == 0:
        return 96
    return 64 if page_size >= 4 and page_size % 64 == 0 else None


def prefer_latent_tcgen05(dtype: torch.dtype, head_dim: int, page_size: int, max_keys: int) -> bool:
    """Whether a step with portions whose rows see up to ``max_keys`` keys runs attention whose values are the keys on the
    tcgen05 kernel: bfloat16 and cached rows in multiples of 16 values up to 256, and enough keys to make up for its later
    start (28 heads over rows of 256 values: 13.4 us against 9.3 for a prompt of 64 tokens, 15.3 against 18.3 for 256, 40
    against 103 for a portion of 16 tokens behind 2,048).  TESSWEAVE_PREFILL_ATTENTION=mma|tcgen05 forces one
    of the two (the latter only for shapes the kernel takes)."""
    import os
    if dtype != torch.bfloat16 or head_dim % 16 or not 16 <= head_dim <= 256 or latent_tcgen05_key_tile(page_size) is None:
        return False
    forced = os.environ.get("TESSWEAVE_PREFILL_ATTENTION")
    if forced in ("mma", "tcgen05"):
        return forced == "tcgen05"
    return max_keys >= LATENT_TCGEN05_MIN_KEYS


def attention_latent_tcgen05(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, pages, n_seqs, max_q_len, n_q_heads,
                             n_kv_heads, head_dim, v_cols, window, scale, skip_single, status, sink: torch.Tensor | None = None,
                             gate: torch.Tensor | None = None) -> None:
    """Prompt attention whose values are the leading ``v_cols`` values of the keys, on the tcgen05 tensor cores
    (csrc/attention_latent_tcgen05.cu).  Of a head's ``head_dim`` outputs the first ``v_cols`` (rounded up to 16) are
    written.  ``sink``, ``gate`` and ``window`` as for ``attention_decode``."""
    _cuda(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, pages, status, sink, gate)
    _gate_check(gate, 0, n_q_heads)
    _attn_common_checks(out, q, block_table, pages, pages, n_q_heads, n_kv_heads, head_dim)
    _score_terms_checks(sink, None, n_q_heads)
    tile = latent_tcgen05_key_tile(pages.shape[2])
    _need(tile is not None and 0 < v_cols <= head_dim and scale > 0, "attention_latent_tcgen05: a page size, value columns or a scale the kernel does not take")
    code = _fn("attention_latent_tcgen05", "tw_attn_latent_tc5", {"TW_HEAD_DIM": head_dim, "TW_V_COLS": -(-v_cols // 16) * 16, "TW_KEY_TILE": tile})(
        _ptr(out), c_int(out.stride(0)), _ptr(q), c_int(q.stride(0)), _ptr(seq_q_start), _ptr(seq_q_len), _ptr(seq_kv_len), _ptr(seq_slot),
        _ptr(block_table), c_int(block_table.shape[1]), _ptr(pages), c_int(n_seqs), c_int(max_q_len), c_int(n_q_heads), c_int(n_kv_heads),
        c_int(pages.shape[2]), c_int(pages.shape[0]), c_int(window), c_float(scale), c_int(1 if skip_single else 0), _ptr(sink), _ptr(gate),
        _ptr(status), _stream())
    _check(code, "attention_latent_tcgen05")


def attention_prefill(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, n_seqs,
                      max_q_len, n_q_heads, n_kv_heads, head_dim, window, scale, skip_single, status,
                      sink: torch.Tensor | None = None, bias_rows: torch.Tensor | None = None,
                      gate: torch.Tensor | None = None) -> None:
    """Flash attention over the paged cache for the requests that bring several tokens.  ``sink``, ``bias_rows``,
    ``gate``, ``window`` and ``v_pages`` that are ``k_pages`` or have rows of another length: as for ``attention_decode``."""
    _cuda(out, q, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, k_pages, v_pages, status, sink, bias_rows, gate)
    _gate_check(gate, 0, n_q_heads)
    _attn_common_checks(out, q, block_table, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim)
    _score_terms_checks(sink, bias_rows, n_q_heads)
    code = _fn("attention_bf16", "tw_attn_prefill", head_size_defines(head_dim, v_pages.shape[3]))(
        _ptr(out), c_int(out.stride(0)), _ptr(q), c_int(q.stride(0)), _ptr(seq_q_start), _ptr(seq_q_len),
        _ptr(seq_kv_len), _ptr(seq_slot), _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages),
        c_int(n_seqs), c_int(max_q_len), c_int(n_q_heads), c_int(n_kv_heads), c_int(k_pages.shape[2]),
        c_int(k_pages.shape[0]), c_int(window), c_float(scale), c_int(1 if skip_single else 0), _ptr(bias_rows),
        c_int(0 if bias_rows is None else bias_rows.shape[1]), _ptr(sink), _ptr(gate), _ptr(status), _stream())
    _check(code, "attention_prefill")


# ---------------------------------------------------------------------------
# matrix products with few rows
# ---------------------------------------------------------------------------
SMALL_M_LIMIT = 8          # rows up to which the weight-streaming kernel is used
_TARGET_WARPS = 2400       # warps in flight that keep the memory system busy


def small_m_supported(x: torch.Tensor, w: torch.Tensor, m: int) -> bool:
    return (x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and 0 < m <= SMALL_M_LIMIT
            and w.shape[1] % 8 == 0 and w.is_contiguous() and x.is_contiguous())


SMALL_M_ROWS_PER_BLOCK = 64      # weight rows of a block of csrc/gemm_smallm.cu (four warps of 16 rows)
SMALL_M_BLOCKS_PER_SM = 5        # how many of its blocks an SM holds


def small_m_split(n: int, k: int, max_slices: int = 12, sms: int | None = None) -> tuple[int, int]:
    """(slices, k per slice): enough slices that rows / 16 * slices warps fill the GPU, each
    slice a multiple of 32 wide and at least 256.  ``max_slices``: the most slices the consumer wants to add
    (the kernel then gives a row tile to two warps where that fills the GPU better).

    All blocks of such a launch are resident at once and share the memory bandwidth about equally, so the launch
    takes as long as the SM with the most blocks: among the slice counts near the one that fills the GPU, the one
    that leaves the SMs most evenly loaded is taken.  Measured on B200, whole decode steps of the 7B-sized model
    (3,584 rows in blocks of 64: 56 blocks per slice): 11 slices = 616 blocks, 4.2 per SM, 3.18 ms; 10 slices =
    560 blocks, 3.8 per SM, 3.13 ms; 13 slices 3.17; 9 slices 3.18; 8 slices (448 blocks, which the kernel doubles:
    6 per SM, two rounds) 3.30; at the 14B sizes (5,120 rows: 80 blocks per slice) 9 slices = 720 blocks 6.88 ms,
    8 slices = 640 blocks 6.93."""
    sms = sms or _SM_COUNT
    tiles = -(-n // 16)
    if tiles >= 1024:          # enough rows to fill the GPU without slices
        return 1, -(-k // 32) * 32
    want = max(1, min(12, max_slices, -(-_TARGET_WARPS // tiles)))
    best = None
    for wanted in range(min(12, max_slices, want + 1), max(0, want - 3), -1):
        kper = max(256, -(-(-(-k // wanted)) // 32) * 32)
        kper = min(kper, -(-k // 32) * 32)
        slices = -(-k // kper)
        blocks = -(-n // SMALL_M_ROWS_PER_BLOCK) * slices
        if blocks * 10 <= sms * 32 and kper >= 512:  # the kernel then gives every row tile to two warps: twice the blocks
            blocks = -(-n // (SMALL_M_ROWS_PER_BLOCK // 2)) * slices
        most = -(-blocks // sms)                     # blocks of the fullest SM
        even = blocks / (most * sms) if most <= SMALL_M_BLOCKS_PER_SM else 0.0
        # fewer slices than wanted only where that evens the load out by a tenth or more
        score = even - 0.03 * abs(want - wanted)
        if best is None or score > best[0]:
            best = (score, slices, kper)
    return best[1], best[2]


def gemm_small_m(out: torch.Tensor, x: torch.Tensor, w: torch.Tensor, m: int, kper: int | None = None,
                 silu_mul_pairs: bool = False, early_dependents: bool = False,
                 prefetch: torch.Tensor | None = None, bias: torch.Tensor | None = None, act: int | None = None) -> None:
    """out[:m] = x[:m] @ w.T for m <= 64 rows.  ``out`` is bf16 or fp32 [>=m, n]; or, when the
    product is split over k (kper < k), fp32 slices [slices, m, n]; or, with ``silu_mul_pairs``
    (rows of w in groups of eight gates and their eight ups), bf16 [>=m, n / 2] = act(gate) * up (silu by default).
    ``bias`` (bf16 [n], in the order of the rows of w) is added first, of a split product to slice 0; without pairs an
    ``act`` is applied to every value (not to slices).
    ``early_dependents``: the kernel launched next may become resident while this one runs (it waits for
    the result itself); worth it when that kernel is small.  ``prefetch``: a contiguous, 16-byte aligned tensor
    that the kernel after this one streams; the blocks ask for it to be brought into L2 when their own stream ends."""
    _cuda(out, x, w, bias)
    if prefetch is not None:
        _need(prefetch.is_cuda and prefetch.is_contiguous(), "gemm_small_m: the tensor to prefetch must be contiguous")
    n, k = w.shape
    _bias_check(bias, n, x.dtype, "gemm_small_m")
    act = (ACT_SILU if silu_mul_pairs else ACT_NONE) if act is None else act
    _need(x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.is_contiguous() and x.is_contiguous()
          and x.shape[1] == k and k % 8 == 0 and m <= 64, "gemm_small_m: bf16 operands, k a multiple of 8, m <= 64")
    kper = kper or -(-k // 32) * 32
    split = -(-k // kper)
    if silu_mul_pairs:
        _need(split == 1 and n % 16 == 0 and out.dtype == torch.bfloat16 and out.dim() == 2 and out.stride(1) == 1
              and out.shape[0] >= m and out.shape[1] == n // 2, "gemm_small_m: bad fused silu output")
        mode, stride = 3, out.stride(0)
    elif split > 1:
        _need(out.dtype == torch.float32 and out.dim() == 3 and out.shape[0] == split and out.shape[1] == m
              and out.shape[2] == n and out.is_contiguous(), "gemm_small_m: split output must be fp32 [slices, m, n]")
        mode, stride = 2, n
    else:
        _need(out.dim() == 2 and out.stride(1) == 1 and out.shape[0] >= m and out.shape[1] == n
              and out.dtype in (torch.bfloat16, torch.float32), "gemm_small_m: bad output")
        mode, stride = (0 if out.dtype == torch.bfloat16 else 1), out.stride(0)
    if early_dependents:
        mode |= 16          # the kernel after this one may become resident while this one runs
    code = _fn("gemm_smallm", "tw_gemm_smallm")(_ptr(w), _ptr(x), c_int(m), c_int(n), c_int(k), c_int(kper), _ptr(out),
                                                c_int(mode), c_int(stride), _ptr(bias), c_int(act), _ptr(prefetch),
                                                ctypes.c_longlong(prefetch.numel() * prefetch.element_size()
                                                                  if prefetch is not None else 0), _stream())
    _check(code, "gemm_small_m")


# ---------------------------------------------------------------------------
# matrix products of prompt steps on pairs of thread blocks
# ---------------------------------------------------------------------------
PAIR_MIN_M = 768           # rows from which the fused gate/up product may run on block pairs


def pair_tiles_efficiency(m: int, n: int, sms: int | None = None) -> float:
    """The share of the block pairs' time that is useful work: rows padded to tiles of 256, and the 256 x 256 tiles
    dealt to sms / 2 pairs in whole rounds."""
    pairs = max(1, (sms or _SM_COUNT) // 2)
    tiles_m, tiles_n = -(-m // 256), -(-n // 256)
    tiles = tiles_m * tiles_n
    return (m / (tiles_m * 256)) * (tiles / pairs) / -(-tiles // pairs)


def pair_product_preferred(x: torch.Tensor, w: torch.Tensor, m: int) -> bool:
    """Whether the gate/up product with the SiLU.mul epilogue runs on ``gemm_tcgen05_pair``.  Measured on B200
    against the library's product plus the separate SiLU.mul kernel: at 37,888 x 3,584 the pairs take 155.7 /
    200.5 / 280.4 / 387 us at 768 / 1,024 / 1,536 / 2,048 rows against 156.2 / 204.8 / 298.0 / 396, but 146.8
    against 124.0 at 544 rows (padded to 768) and 109.6 against 108.1 at 512; at 27,648 x 5,120 they lose where
    the tiles do not fill whole rounds of pairs (1,280 rows: 271.9 against 260.7).  So: from 768 rows, and only
    where padding and rounds leave at least 93 % of the pairs' time useful.  TESSWEAVE_PAIR_GEMM=0 keeps the library,
    =force takes the pairs for every shape beyond 64 rows."""
    import os
    choice = os.environ.get("TESSWEAVE_PAIR_GEMM", "1")
    if choice == "0":
        return False
    takes = (x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.shape[0] % 16 == 0
             and w.shape[1] % 8 == 0 and x.is_contiguous() and w.is_contiguous())
    if choice == "force":          # every shape the kernel takes (tests run whole models through it this way)
        return takes and m > 64
    return takes and m >= PAIR_MIN_M and pair_tiles_efficiency(m, w.shape[0]) >= 0.93


def gemm_tcgen05_pair(out: torch.Tensor, x: torch.Tensor, w: torch.Tensor, m: int, status: torch.Tensor,
                      silu_mul_pairs: bool = False, bias: torch.Tensor | None = None, act: int | None = None) -> None:
    """out[:m] = x[:m] @ w.T for many rows, on pairs of thread blocks (tcgen05.mma.cta_group::2,
    256 x 256 tiles).  ``out`` is bf16 or fp32 [>=m, n]; with ``silu_mul_pairs`` (rows of w in
    groups of eight gates and their eight ups) it is bf16 [>=m, n / 2] = act(gate) * up.  ``bias`` and ``act``: as for
    ``gemm_small_m``."""
    _cuda(out, x, w, status, bias)
    n, k = w.shape
    _bias_check(bias, n, x.dtype, "gemm_tcgen05_pair")
    act = (ACT_SILU if silu_mul_pairs else ACT_NONE) if act is None else act
    _need(x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.is_contiguous() and x.is_contiguous()
          and x.shape[1] == k and k % 8 == 0, "gemm_tcgen05_pair: contiguous bf16 operands, k a multiple of 8")
    _need(x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0, "gemm_tcgen05_pair: operands must be 16-byte aligned")
    if silu_mul_pairs:
        _need(n % 16 == 0 and out.dtype == torch.bfloat16 and out.dim() == 2 and out.stride(1) == 1 and out.shape[0] >= m
              and out.shape[1] == n // 2 and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0,
              "gemm_tcgen05_pair: the SiLU.mul output must be bf16 [m, n / 2] with 16-byte aligned rows")
        mode = 3
    else:
        _need(out.dim() == 2 and out.stride(1) == 1 and out.shape[0] >= m and out.shape[1] == n
              and out.dtype in (torch.bfloat16, torch.float32), "gemm_tcgen05_pair: bad output")
        mode = 0 if out.dtype == torch.bfloat16 else 1
    code = _fn("gemm_tcgen05_pair", "tw_gemm_tcgen05_pair")(_ptr(x), _ptr(w), c_int(m), c_int(n), c_int(k), _ptr(out),
                                                            c_int(mode), c_int(out.stride(0)), _ptr(bias), c_int(act), _ptr(status),
                                                            _stream())
    _check(code, "gemm_tcgen05_pair")


# ---------------------------------------------------------------------------
# matrix products of decode steps with more requests than the small-M kernel takes
# ---------------------------------------------------------------------------
STREAM_MIN_M, STREAM_MAX_M = 9, 128     # rows the persistent weight-streaming tcgen05 kernel takes
STREAM_MIN_WEIGHTS = 48_000_000         # elements of w from which it is the product path


def stream_product_preferred(x: torch.Tensor, w: torch.Tensor, m: int) -> bool:
    """Whether a product of ``m`` rows runs on ``gemm_tcgen05_stream`` (persistent, the weights as the 128-row
    operand): 9 to 64 rows and a large matrix.  Measured on B200 at 7B layer sizes, 16 / 64 rows: down 25.9 / 28.1
    us against the library's 28.9 / 31.1, gate/up with SiLU.mul 47.5 / 51.7 against 46.6 / 48.1 plus 2.5 / 3.5 for
    the separate SiLU.mul kernel, logits 171 / 181 against 179 / 183; the smaller q/k/v and o_proj products
    (8.8 / 10.7 against 8.6 / 8.9) stay with the library, whose split over k is reduced inside its kernel.
    TESSWEAVE_STREAM_GEMM=0 keeps the library everywhere; TESSWEAVE_STREAM_MAX_M and TESSWEAVE_STREAM_MIN_WEIGHTS
    move the bounds."""
    import os
    if os.environ.get("TESSWEAVE_STREAM_GEMM", "1") == "0":
        return False
    top = min(STREAM_MAX_M, int(os.environ.get("TESSWEAVE_STREAM_MAX_M", "64")))
    least = int(os.environ.get("TESSWEAVE_STREAM_MIN_WEIGHTS", str(STREAM_MIN_WEIGHTS)))
    return (x.is_cuda and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and STREAM_MIN_M <= m <= top
            and w.numel() >= least and w.shape[1] % 8 == 0 and x.is_contiguous() and w.is_contiguous()
            and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


_stream_sms: list[int] = [0]


def _stream_sm_count() -> int:
    if not _stream_sms[0]:
        _stream_sms[0] = int(_fn("gemm_tcgen05_stream", "tw_gemm_tcgen05_stream_sm_count")())
    return _stream_sms[0]


def stream_whole_k_balanced(n: int, sms: int | None = None) -> bool:
    """Whether the 128-row tiles of a matrix of ``n`` rows, not split over k (the SiLU.mul epilogue needs whole
    sums), keep the persistent kernel's blocks evenly busy: 296 tiles on 148 SMs do (two each), 216 do not (68
    blocks get two, 80 one; the 14B gate/up product measured slower than the library that way)."""
    sms = sms or _stream_sm_count()
    tiles = -(-n // 128)
    return tiles / sms >= 0.85 * -(-tiles // sms)


def stream_split_gate_up_enabled() -> bool:
    """TESSWEAVE_STREAM_SPLIT_GATE_UP=1: a gate/up product whose row tiles alone do not balance (14B: 216 tiles)
    runs on the persistent kernel in slices over k that the SiLU.mul kernel adds.  Off by default: measured at 14B
    layer sizes a decode step is 1 % shorter with it at batch 12 and 24 and 2.5 % longer at batch 32, where the
    library's product is at its best."""
    import os
    return os.environ.get("TESSWEAVE_STREAM_SPLIT_GATE_UP", "0") == "1"


def stream_split(n: int, k: int, allow: bool = True, sms: int | None = None) -> tuple[int, int]:
    """(slices, k per slice) for the persistent kernel: its work items are (128-row tile of w, slice of k), dealt
    round robin to one block per SM.  The choice minimises the k-blocks of the busiest block, each item charged
    four more for its start and its result; up to 12 slices."""
    kbs = -(-k // 64)
    if not allow:
        return 1, kbs * 64
    sms = sms or _stream_sm_count()
    tiles = -(-n // 128)
    best = None
    for want in range(1, 13):
        per = -(-kbs // want)
        real = -(-kbs // per)
        cost = -(-tiles * real // sms) * (per + 4)
        if best is None or cost < best[0]:
            best = (cost, real, per * 64)
    return best[1], best[2]


def gemm_tcgen05_stream(out: torch.Tensor, x: torch.Tensor, w: torch.Tensor, m: int, status: torch.Tensor,
                        kper: int | None = None, silu_mul_pairs: bool = False, early_dependents: bool = False,
                        prefetch: torch.Tensor | None = None, bias: torch.Tensor | None = None, act: int | None = None) -> None:
    """out[:m] = x[:m] @ w.T for up to 128 rows on the 5th-generation tensor cores, the weights streamed once by a
    persistent kernel.  ``out`` is bf16 or fp32 [>=m, n]; fp32 slices [slices, m, n] when ``kper`` (a multiple of
    64) is less than k; with ``silu_mul_pairs`` (rows of w in groups of eight gates and their eight ups) bf16
    [>=m, n / 2] = act(gate) * up.  ``bias`` and ``act``: as for ``gemm_small_m``.  ``prefetch``: a contiguous, 16-byte aligned tensor that the kernel after
    this one streams; a block asks for its share of it to be brought into L2 once its own last copy is issued."""
    _cuda(out, x, w, status, bias)
    _bias_check(bias, w.shape[0], x.dtype, "gemm_tcgen05_stream")
    act = (ACT_SILU if silu_mul_pairs else ACT_NONE) if act is None else act
    if prefetch is not None:
        _need(prefetch.is_cuda and prefetch.is_contiguous(), "gemm_tcgen05_stream: the tensor to prefetch must be contiguous")
    n, k = w.shape
    _need(x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.is_contiguous() and x.is_contiguous()
          and x.shape[1] == k and k % 8 == 0 and 0 < m <= STREAM_MAX_M and x.shape[0] >= m,
          "gemm_tcgen05_stream: contiguous bf16 operands, k a multiple of 8, up to 128 rows")
    _need(x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0, "gemm_tcgen05_stream: operands must be 16-byte aligned")
    kper = kper or -(-k // 64) * 64
    _need(kper % 64 == 0, "gemm_tcgen05_stream: k per slice must be a multiple of 64")
    split = -(-k // kper)
    if silu_mul_pairs:
        _need(split == 1 and n % 16 == 0 and out.dtype == torch.bfloat16 and out.dim() == 2 and out.stride(1) == 1
              and out.shape[0] >= m and out.shape[1] == n // 2, "gemm_tcgen05_stream: bad fused SiLU.mul output")
        mode, stride = 3, out.stride(0)
    elif split > 1:
        _need(out.dtype == torch.float32 and out.dim() == 3 and tuple(out.shape) == (split, m, n) and out.is_contiguous(),
              "gemm_tcgen05_stream: split output must be fp32 [slices, m, n]")
        mode, stride = 2, n
    else:
        _need(out.dim() == 2 and out.stride(1) == 1 and out.shape[0] >= m and out.shape[1] == n
              and out.dtype in (torch.bfloat16, torch.float32), "gemm_tcgen05_stream: bad output")
        mode, stride = (0 if out.dtype == torch.bfloat16 else 1), out.stride(0)
    if early_dependents:
        mode |= 16          # the kernel after this one may become resident while this one runs
    # the token rows the kernel reads: exactly m (rows beyond are filled with zeros by the copy engine)
    code = _fn("gemm_tcgen05_stream", "tw_gemm_tcgen05_stream")(_ptr(x), _ptr(w), c_int(m), c_int(n), c_int(k), c_int(kper),
                                                                _ptr(out), c_int(mode), c_int(stride), _ptr(bias), c_int(act), _ptr(status),
                                                                _ptr(prefetch), ctypes.c_longlong(
                                                                    prefetch.numel() * prefetch.element_size()
                                                                    if prefetch is not None else 0), _stream())
    _check(code, "gemm_tcgen05_stream")


# ---------------------------------------------------------------------------
# pieces of mixers that are not attention over a cache: recurrences with a matrix state, token shift
# ---------------------------------------------------------------------------
RECURRENCE_RETENTION, RECURRENCE_WKV, RECURRENCE_MLSTM, RECURRENCE_DELTA, RECURRENCE_GLA, RECURRENCE_SSD = 0, 1, 2, 3, 4, 5
RECURRENCE_MAX_KEY_DIM = 256      # a thread keeps a column of the state in registers (beyond 128 it spills)


def recurrence_state_numel(mode: int, heads: int, key_dim: int, value_dim: int) -> int:
    """fp32 values a request's state takes: per head S [Dk, Dv]; the mLSTM rule adds its normaliser as one more
    column and its running maximum."""
    if mode == RECURRENCE_MLSTM:
        return heads * (key_dim * (value_dim + 1) + 1)
    return heads * key_dim * value_dim


def linear_recurrence(mode: int, out: torch.Tensor, den: torch.Tensor | None, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor,
                      state: torch.Tensor, positions: torch.Tensor, seq_slot: torch.Tensor, seq_q_start: torch.Tensor,
                      seq_q_len: torch.Tensor, n_seqs: int, heads: int, key_dim: int, value_dim: int, write_state: bool = True,
                      pre: torch.Tensor | None = None, p0: torch.Tensor | None = None, p1: torch.Tensor | None = None,
                      inv_freq: torch.Tensor | None = None, rot_dims: int = 0, q_scale: float = 1.0, k_scale: float = 1.0,
                      cap: float = 1.0, tail: torch.Tensor | None = None, tail_offset: int = 0, max_q_len: int = 1 << 30,
                      write_pre: torch.Tensor | None = None, channel_decay: bool = False, qk_group: int = 1,
                      p2: torch.Tensor | None = None) -> None:
    """Walk every request's rows of the step through its matrix state (csrc/linear_recurrence.cu): ``out`` fp32
    [rows, heads * value_dim] receives the raw outputs, ``den`` fp32 [rows, heads] the mLSTM denominators.  q, k, v are
    column slices of the projected rows (heads side by side).  ``pre``: fp32 rows the rule needs beside them (wkv:
    the projected decay [rows, heads * key_dim]; mlstm: the gates' pre-activations [rows, 2 * heads]); ``p0`` / ``p1``
    fp32 constants (wkv: decay offset and bonus; retention: decay per head; mlstm: gate biases).  ``tail``: rows whose
    last one per request is copied into the state behind the heads (wkv's token shift), at ``tail_offset``.
    ``max_q_len``: the longest portion of the step (a hint: steps of single tokens launch smaller blocks).
    The delta rule takes fp32 q, k, v that are ready to use, ``pre`` the projected decay ([rows, heads * key_dim] with
    ``channel_decay``, else [rows, heads]), ``p0`` the log of each head's rate [heads], ``p1`` the decay's bias (of
    ``pre``'s width), ``write_pre`` the write strength before its sigmoid, fp32 [rows, heads]; ``qk_group`` value heads
    share a head of q and k.  Gated linear attention takes ``pre`` the projected decay [rows, heads * key_dim], ``p0`` its
    bias and ``cap`` the exponent 1 / tau of the sigmoid.  The state-space rule takes q, k, v that are ready to use,
    ``pre`` the projected step size [rows, heads], ``p0`` the log of each head's rate, ``p1`` the step size's bias and ``p2``
    the skip, each [heads]; ``qk_group`` as in the delta rule."""
    _cuda(out, den, q, k, v, state, positions, seq_slot, seq_q_start, seq_q_len, pre, p0, p1, p2, inv_freq, tail, write_pre)
    _need(mode != RECURRENCE_SSD or (pre is not None and pre.stride(1) == 1 and pre.shape[1] >= heads
                                     and all(p is not None and p.numel() == heads and p.is_contiguous() for p in (p0, p1, p2))
                                     and qk_group >= 1 and heads % qk_group == 0),
          "recurrence: the state-space rule needs a projected step size, and a rate, bias and skip per head")
    if mode == RECURRENCE_DELTA:
        width = heads * key_dim if channel_decay else heads
        _need(q.dtype == torch.float32 and pre is not None and p0 is not None and p1 is not None and write_pre is not None
              and write_pre.dtype == torch.float32 and write_pre.stride(1) == 1 and write_pre.shape[1] >= heads
              and pre.stride(1) == 1 and pre.shape[1] >= width and p1.numel() == width and p0.numel() == heads
              and qk_group >= 1 and heads % qk_group == 0,
              "recurrence: the delta rule needs fp32 rows, a projected decay with its rate and bias, and a write strength")
    _need(out.dtype == torch.float32 and out.is_contiguous() and out.shape[1] == heads * value_dim, "recurrence: out must be fp32 [rows, H * Dv]")
    _need(q.dtype == k.dtype == v.dtype and q.stride(1) == k.stride(1) == v.stride(1) == 1, "recurrence: q, k, v of one type, unit column stride")
    _need(state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1, "recurrence: state must be fp32 [slots, numel]")
    _need(0 < key_dim <= 256 and 0 < value_dim <= 256, "recurrence: head sizes must lie in 1..256")
    for t in (pre, p0, p1, p2, inv_freq, den):
        _need(t is None or t.dtype == torch.float32, "recurrence: constants, gates and denominators are fp32")
    _need(mode != RECURRENCE_MLSTM or (den is not None and pre is not None and p0 is not None), "recurrence: mlstm needs gates and a denominator buffer")
    _need(mode != RECURRENCE_WKV or (pre is not None and p0 is not None and p1 is not None and key_dim == value_dim), "recurrence: wkv needs decay rows, offset and bonus")
    _need(mode != RECURRENCE_RETENTION or p0 is not None, "recurrence: retention needs a decay per head")
    _need(mode != RECURRENCE_GLA or (pre is not None and p0 is not None and pre.stride(1) == 1 and pre.shape[1] >= heads * key_dim
                                     and p0.numel() == heads * key_dim and cap > 0),
          "recurrence: gated linear attention needs the projected decay rows, their bias and a positive exponent")
    code = _fn("linear_recurrence", "tw_linear_recurrence", {"TW_DK": key_dim})(
        c_int(mode), _ptr(out), _ptr(den), _ptr(q), c_int(q.stride(0)), _ptr(k), c_int(k.stride(0)), _ptr(v), c_int(v.stride(0)),
        _ptr(pre), c_int(0 if pre is None else pre.stride(0)), _ptr(p0), _ptr(p1), _ptr(p2), _ptr(write_pre),
        c_int(0 if write_pre is None else write_pre.stride(0)), c_int(1 if channel_decay else 0), c_int(qk_group),
        _ptr(inv_freq), c_int(rot_dims),
        c_float(q_scale), c_float(k_scale), c_float(cap), _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(tail),
        c_int(0 if tail is None else tail.stride(0)), c_int(0 if tail is None else tail.shape[1]), ctypes.c_longlong(tail_offset),
        _ptr(positions), _ptr(seq_slot), _ptr(seq_q_start), _ptr(seq_q_len), c_int(n_seqs), c_int(heads), c_int(key_dim),
        c_int(value_dim), c_int(1 if write_state else 0), c_int(max_q_len), c_int(dtype_code(q.dtype)), _stream())
    _check(code, "linear_recurrence")


STATE_SPACE_CHUNK_STATES = (16, 32, 64, 128, 256)
STATE_SPACE_CHUNK_MIN_TOKENS = 12       # 112 heads of 128 x 64, one request / eight: 7 / 42 us in chunks, token by token 9 / 37 us for 12


def state_space_chunks_supported(dtype: torch.dtype, state_dim: int, value_dim: int, channels: int, max_q_len: int) -> bool:
    """Whether a step whose longest portion has ``max_q_len`` tokens runs the state-space recurrence in chunks on the
    tensor cores: bfloat16 rows, state sizes and values the tiles take, and more than a few tokens.
    TESSWEAVE_STATE_SPACE=tokens|chunks forces one of the two (the latter only for sizes the kernel takes)."""
    import os
    if dtype != torch.bfloat16 or state_dim not in STATE_SPACE_CHUNK_STATES or value_dim % 16 or channels % 8:
        return False
    forced = os.environ.get("TESSWEAVE_STATE_SPACE")
    if forced in ("tokens", "chunks"):
        return forced == "chunks"
    return max_q_len >= STATE_SPACE_CHUNK_MIN_TOKENS


def state_space_slice(heads: int, n_seqs: int, value_dim: int, sms: int = 148) -> int:
    """Values of a head that a block of the chunked kernel serves: 64 where they divide, less where that would leave more
    than half of the SMs without a block (a slice repeats the products that do not depend on the values)."""
    sizes = [d for d in (64, 32, 16) if value_dim % d == 0]
    for d in sizes:
        if heads * n_seqs * (value_dim // d) > sms // 2 or d == sizes[-1]:
            return d
    raise KernelError(f"the chunked state-space kernel takes values in multiples of 16, not {value_dim}")


def state_space_chunks(out: torch.Tensor, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, pre: torch.Tensor, rate_log: torch.Tensor,
                       dt_bias: torch.Tensor, skip: torch.Tensor, state: torch.Tensor, seq_slot: torch.Tensor, seq_q_start: torch.Tensor,
                       seq_q_len: torch.Tensor, n_seqs: int, heads: int, state_dim: int, value_dim: int, qk_group: int,
                       write_state: bool = True, slice_dim: int | None = None) -> None:
    """``linear_recurrence`` with the state-space rule over portions of a prompt, 64 tokens at a time on the tensor cores
    (csrc/state_space.cu): same operands and state, bfloat16 q, k, v."""
    _cuda(out, q, k, v, pre, rate_log, dt_bias, skip, state, seq_slot, seq_q_start, seq_q_len)
    _need(out.dtype == torch.float32 and out.is_contiguous() and out.shape[1] == heads * value_dim, "state_space_chunks: out must be fp32 [rows, H * Dv]")
    _need(all(t.dtype == torch.bfloat16 and t.stride(1) == 1 for t in (q, k, v)) and heads % qk_group == 0
          and q.shape[1] == k.shape[1] == heads // qk_group * state_dim and v.shape[1] == heads * value_dim,
          "state_space_chunks: q, k, v must be bf16 rows of their heads")
    _need(pre.dtype == torch.float32 and pre.stride(1) == 1 and pre.shape[1] >= heads
          and all(p.dtype == torch.float32 and p.numel() == heads and p.is_contiguous() for p in (rate_log, dt_bias, skip)),
          "state_space_chunks: fp32 step sizes [rows, H] and constants [H]")
    _need(state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1 and state.shape[1] >= heads * state_dim * value_dim,
          "state_space_chunks: the state must be fp32 [slots, numel]")
    code = _fn("state_space", "tw_state_space_chunks", {"TW_DK": state_dim})(
        _ptr(out), _ptr(q), c_int(q.stride(0)), _ptr(k), c_int(k.stride(0)), _ptr(v), c_int(v.stride(0)), _ptr(pre), c_int(pre.stride(0)),
        _ptr(rate_log), _ptr(dt_bias), _ptr(skip), _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(seq_slot), _ptr(seq_q_start),
        _ptr(seq_q_len), c_int(n_seqs), c_int(heads), c_int(state_dim), c_int(value_dim), c_int(qk_group),
        c_int(slice_dim or state_space_slice(heads, n_seqs, value_dim)), c_int(1 if write_state else 0), _stream())
    _check(code, "state_space_chunks")


GATE_NONE, GATE_SILU, GATE_SIGMOID = 0, 1, 2


def head_norm_gate(out: torch.Tensor, raw: torch.Tensor, den: torch.Tensor | None, weight: torch.Tensor | None,
                   gate: torch.Tensor | None, act: int, eps: float, n_rows: int, heads: int, value_dim: int) -> None:
    """out[row, h] = rms_h(raw[row, h] / den[row, h]) * weight[h] * act(gate[row, h]): the norm over each head of a
    recurrence's fp32 output, the optional weight and gate, rounded to the type of ``out``."""
    _cuda(out, raw, den, weight, gate)
    _need(raw.dtype == torch.float32 and raw.is_contiguous() and raw.shape[1] == heads * value_dim, "head_norm_gate: raw must be fp32 [rows, H * Dv]")
    _need(out.stride(1) == 1 and out.shape[1] >= heads * value_dim, "head_norm_gate: bad output")
    _need(weight is None or (weight.dtype == torch.float32 and weight.numel() == heads * value_dim), "head_norm_gate: weight fp32 [H * Dv]")
    _need(den is None or (den.dtype == torch.float32 and den.is_contiguous()), "head_norm_gate: den fp32 [rows, H]")
    _need((act == GATE_NONE) == (gate is None) and (gate is None or (gate.dtype == out.dtype and gate.stride(1) == 1)),
          "head_norm_gate: a gate of the output's type exactly when an activation is named")
    code = _fn("recurrent", "tw_head_norm_gate")(
        _ptr(out), c_int(out.stride(0)), _ptr(raw), _ptr(den), _ptr(weight), _ptr(gate), c_int(0 if gate is None else gate.stride(0)),
        c_int(act), c_float(eps), c_int(n_rows), c_int(heads), c_int(value_dim), c_int(dtype_code(out.dtype)), _stream())
    _check(code, "head_norm_gate")


def gate_part_norm(out: torch.Tensor, raw: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, act: int, eps: float, n_rows: int,
                   parts: int) -> None:
    """u = raw * act(gate) (fp32 ``raw`` [rows, width], ``gate`` a column slice of rows of the output's type); each of the
    ``parts`` equal parts of a row of u is divided by its own root mean square; times ``weight`` (fp32 [width])."""
    _cuda(out, raw, weight, gate)
    width = raw.shape[1]
    _need(raw.dtype == torch.float32 and raw.is_contiguous() and parts >= 1 and width % parts == 0, "gate_part_norm: raw must be fp32 rows of equal parts")
    _need(out.stride(1) == 1 and out.shape[1] == width and gate.dtype == out.dtype and gate.stride(1) == 1 and gate.shape[1] == width
          and min(out.shape[0], raw.shape[0], gate.shape[0]) >= n_rows, "gate_part_norm: gate and output rows of one type and raw's width")
    _need(weight.dtype == torch.float32 and weight.is_contiguous() and weight.numel() == width, "gate_part_norm: weight fp32 [width]")
    _need(act in (GATE_SILU, GATE_SIGMOID), "gate_part_norm: the activation is silu or sigmoid")
    code = _fn("recurrent", "tw_gate_part_norm")(
        _ptr(out), c_int(out.stride(0)), _ptr(raw), _ptr(weight), _ptr(gate), c_int(gate.stride(0)), c_int(act), c_float(eps),
        c_int(n_rows), c_int(width), c_int(parts), c_int(dtype_code(out.dtype)), _stream())
    _check(code, "gate_part_norm")


def token_shift_mix(out: torch.Tensor, h: torch.Tensor, mu: torch.Tensor, state: torch.Tensor, state_offset: int,
                    seq_of_token: torch.Tensor, seq_slot: torch.Tensor, seq_q_start: torch.Tensor, n_rows: int) -> None:
    """out[m, row] = h[row] + (h[row - 1] - h[row]) * mu[m] for every blend m; the row before a request's first row
    of this step is read from the request's state (fp32 [slots, numel], ``width`` values at ``state_offset``)."""
    _cuda(out, h, mu, state, seq_of_token, seq_slot, seq_q_start)
    n_mix, width = mu.shape
    _need(out.is_contiguous() and out.dim() == 3 and out.shape[0] == n_mix and out.shape[1] >= n_rows and out.shape[2] == width
          and out.dtype == h.dtype and h.stride(1) == 1 and h.shape[1] == width, "token_shift_mix: out [mixes, rows, width] of h's type")
    _need(mu.dtype == torch.float32 and mu.is_contiguous() and state.dtype == torch.float32 and state.stride(1) == 1,
          "token_shift_mix: mu and state are fp32")
    code = _fn("recurrent", "tw_token_shift_mix")(
        _ptr(out), ctypes.c_longlong(out.stride(0)), _ptr(h), c_int(h.stride(0)), _ptr(mu), _ptr(state),
        ctypes.c_longlong(state.stride(0)), ctypes.c_longlong(state_offset), _ptr(seq_of_token), _ptr(seq_slot), _ptr(seq_q_start),
        c_int(n_rows), c_int(width), c_int(n_mix), c_int(dtype_code(h.dtype)), _stream())
    _check(code, "token_shift_mix")


def tanh_rows(x: torch.Tensor) -> None:
    """tanh of every element of a contiguous tensor, in place."""
    _cuda(x)
    _need(x.is_contiguous(), "tanh_rows: contiguous operand")
    code = _fn("recurrent", "tw_tanh_rows")(_ptr(x), ctypes.c_longlong(x.numel()), c_int(dtype_code(x.dtype)), _stream())
    _check(code, "tanh_rows")


# ---------------------------------------------------------------------------
# hyper-connections
# ---------------------------------------------------------------------------
HYPER_MAX_COPIES = 16


def hyper_step(streams: torch.Tensor, n_rows: int, init: torch.Tensor | None = None, y: torch.Tensor | None = None,
               mix: torch.Tensor | None = None, out_coef: torch.Tensor | None = None, in_coef: torch.Tensor | None = None,
               norm_weight: torch.Tensor | None = None, eps: float = 0.0, h_out: torch.Tensor | None = None,
               sum_out: torch.Tensor | None = None) -> None:
    """One pass over the copies of the residual stream (fp32 [rows, copies, width], in place), doing in this order what
    is given: start every copy from ``init``; write a sub-layer's output ``y`` (x_t <- sum_s mix[s, t] x_s +
    out_coef[t] y); read for the next sub-layer (``h_out`` = rmsnorm(sum_s in_coef[s] x_s) * norm_weight); sum the copies
    into ``sum_out``."""
    _cuda(streams, init, y, mix, out_coef, in_coef, norm_weight, h_out, sum_out)
    _need(streams.dtype == torch.float32 and streams.is_contiguous() and streams.dim() == 3 and streams.shape[0] >= n_rows,
          "hyper_step: the copies must be contiguous fp32 [rows, copies, width]")
    copies, width = streams.shape[1], streams.shape[2]
    _need(copies <= HYPER_MAX_COPIES, f"hyper_step: at most {HYPER_MAX_COPIES} copies of the stream")
    for t, shape in ((init, (width,)), (sum_out, (width,))):
        _need(t is None or (t.dtype == torch.float32 and t.is_contiguous() and tuple(t.shape[1:]) == shape and t.shape[0] >= n_rows),
              "hyper_step: init and sum_out are fp32 [rows, width]")
    _need(y is None or (mix is not None and out_coef is not None and y.is_contiguous() and y.shape[1] == width and y.shape[0] >= n_rows
                        and mix.dtype == out_coef.dtype == torch.float32 and mix.is_contiguous() and mix.numel() == copies * copies
                        and out_coef.numel() == copies), "hyper_step: a write needs y [rows, width], mix [copies, copies] and out_coef [copies]")
    _need(in_coef is None or (h_out is not None and norm_weight is not None and in_coef.dtype == norm_weight.dtype == torch.float32
                              and in_coef.numel() == copies and norm_weight.numel() == width and h_out.is_contiguous()
                              and h_out.shape[1] == width and h_out.shape[0] >= n_rows),
          "hyper_step: a read needs in_coef [copies], a norm weight [width] and h_out [rows, width]")
    _need(y is None or h_out is None or y.dtype == h_out.dtype, "hyper_step: y and h_out of one type")
    dtype = y.dtype if y is not None else (h_out.dtype if h_out is not None else torch.float32)
    code = _fn("hyper_connections", "tw_hyper_step")(
        _ptr(streams), _ptr(init), _ptr(y), _ptr(mix), _ptr(out_coef), _ptr(in_coef), _ptr(norm_weight), c_float(eps), _ptr(h_out),
        _ptr(sum_out), c_int(n_rows), c_int(width), c_int(copies), c_int(dtype_code(dtype)), _stream())
    _check(code, "hyper_step")


# ---------------------------------------------------------------------------
# attention mixers with keys and values of different sizes, or a position encoding no fused kernel takes
# ---------------------------------------------------------------------------
def add_bias_rows(rows: torch.Tensor, bias: torch.Tensor, n_rows: int) -> None:
    """rows[:, :len(bias)] += bias, in place."""
    _cuda(rows, bias)
    _need(rows.stride(1) == 1 and bias.dtype == torch.float32 and bias.numel() <= rows.shape[1], "add_bias_rows: bad operands")
    code = _fn("elementwise", "tw_add_bias_rows")(_ptr(rows), c_int(rows.stride(0)), _ptr(bias), c_int(n_rows), c_int(bias.numel()),
                                                  c_int(dtype_code(rows.dtype)), _stream())
    _check(code, "add_bias_rows")


def kv_store(rows: torch.Tensor, k_col: int, v_col: int, positions: torch.Tensor, seq_of_token: torch.Tensor, seq_slot: torch.Tensor,
             block_table: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor | None, n_tokens: int,
             status: torch.Tensor) -> None:
    """Copy the keys (columns from ``k_col``) and values (from ``v_col``) of the step's packed rows into their pages;
    key pages are [pages, kv_heads, page, Dk], value pages [pages, kv_heads, page, Dv].  ``v_pages`` None: only the keys
    are stored (a mixer whose values are its keys keeps one set of pages)."""
    _cuda(rows, positions, seq_of_token, seq_slot, block_table, k_pages, v_pages, status)
    _need(rows.stride(1) == 1 and rows.dtype == k_pages.dtype and k_pages.is_contiguous(), "kv_store: pages must be contiguous and of the rows' type")
    _need(v_pages is None or (v_pages.dtype == rows.dtype and v_pages.is_contiguous() and k_pages.shape[:3] == v_pages.shape[:3]),
          "kv_store: value pages must be contiguous, of the rows' type and as many as the key pages")
    _need(block_table.dtype == torch.int32 and block_table.is_contiguous(), "kv_store: bad block table")
    code = _fn("elementwise", "tw_kv_store")(
        _ptr(rows), c_int(rows.stride(0)), c_int(k_col), c_int(v_col), _ptr(positions), _ptr(seq_of_token), _ptr(seq_slot),
        _ptr(block_table), c_int(block_table.shape[1]), _ptr(k_pages), _ptr(v_pages), c_int(n_tokens), c_int(k_pages.shape[1]),
        c_int(k_pages.shape[3]), c_int(0 if v_pages is None else v_pages.shape[3]), c_int(k_pages.shape[2]), c_int(k_pages.shape[0]),
        c_int(dtype_code(rows.dtype)), _ptr(status), _stream())
    _check(code, "kv_store")


# ---------------------------------------------------------------------------
# routed feed-forward
# ---------------------------------------------------------------------------
def moe_route(chosen: torch.Tensor, weight: torch.Tensor, shared_gate: torch.Tensor | None, h: torch.Tensor, w_router: torch.Tensor,
              b_router: torch.Tensor | None, w_shared_gate: torch.Tensor | None, n_rows: int, top: int,
              score_all: bool = False, correction: torch.Tensor | None = None, weight_scale: float = 1.0,
              renormalise: bool = False, groups: tuple[int, int] | None = None) -> None:
    """Per row: the ``top`` experts with the largest fp32 logits ``w_router h + b_router`` (int32 [rows, top]), the
    softmax over those logits alone (fp32 [rows, top]), and ``sigmoid(w_shared_gate . h)`` (fp32 [rows]) if asked.
    With ``score_all`` the scores are the softmax over every router output, the choice goes by score + ``correction``
    (fp32 [outputs], may be None) and the weights are the chosen scores times ``weight_scale``, not renormalised -- or, with ``renormalise``, the chosen scores over their
    sum (+ 1e-20) times ``weight_scale``.  ``groups`` = (count, keep): the outputs form ``count`` groups of as many consecutive outputs
    and only those of the ``keep`` groups with the largest best score may be chosen."""
    _cuda(chosen, weight, shared_gate, h, w_router, b_router, w_shared_gate, correction)
    experts, width = w_router.shape
    _need(correction is None or (score_all and correction.dtype == torch.float32 and correction.numel() == experts
                                 and correction.is_contiguous()), "moe_route: the correction is fp32 [router outputs] and goes with score_all")
    count, keep = groups if groups is not None else (0, 0)
    _need((groups is None and not renormalise) or score_all, "moe_route: groups and renormalised weights go with score_all")
    _need(groups is None or (0 < keep <= count and experts % count == 0 and keep * (experts // count) >= top),
          "moe_route: the kept groups must be some of equal groups, and hold enough outputs")
    _need(chosen.dtype == torch.int32 and weight.dtype == torch.float32 and chosen.is_contiguous() and weight.is_contiguous()
          and chosen.shape[1] == weight.shape[1] == top and chosen.shape[0] >= n_rows, "moe_route: chosen int32 / weight fp32 [rows, top]")
    _need(h.stride(1) == 1 and h.shape[1] == width and h.dtype == w_router.dtype and w_router.is_contiguous() and 0 < top <= experts,
          "moe_route: bad operands")
    _need(b_router is None or (b_router.dtype == torch.float32 and b_router.numel() == experts), "moe_route: bias fp32 [experts]")
    _need((w_shared_gate is None) == (shared_gate is None) and (w_shared_gate is None or (
        w_shared_gate.dtype == h.dtype and w_shared_gate.numel() == width and w_shared_gate.is_contiguous() and shared_gate.dtype == torch.float32)),
        "moe_route: the shared gate needs a vector of the activations' type and an fp32 output")
    code = _fn("moe", "tw_moe_route")(_ptr(chosen), _ptr(weight), _ptr(shared_gate), _ptr(h), c_int(h.stride(0)), _ptr(w_router),
                                      _ptr(b_router), _ptr(w_shared_gate), c_int(n_rows), c_int(width), c_int(experts), c_int(top),
                                      c_int((2 if renormalise else 1) if score_all else 0), _ptr(correction), c_float(weight_scale),
                                      c_int(count), c_int(keep),
                                      c_int(dtype_code(h.dtype)), _stream())
    _check(code, "moe_route")


GLU_SILU, GLU_CLAMPED = 0, 1      # what an expert makes of its gate and up products (csrc/moe.cu: tw_glu)


def moe_gate_up(act: torch.Tensor, h: torch.Tensor, w_gate_up: torch.Tensor, chosen: torch.Tensor, n_rows: int,
                glu: int = GLU_SILU, limit: float = 0.0, alpha: float = 1.0) -> None:
    """act[row, j] = silu(Wg_e h[row]) * (Wu_e h[row]) for the j-th chosen expert e of the row;
    ``w_gate_up`` is [experts, 2, ff, width] (a gate matrix followed by its up matrix).  ``GLU_CLAMPED``: with
    g = min(gate, limit) and u = clamp(up, -limit, limit) the activation is g * sigmoid(alpha g) * (u + 1).  A chosen
    index beyond the experts (an expert without matrices) leaves its row of ``act`` untouched."""
    _cuda(act, h, w_gate_up, chosen)
    experts, two, ff, width = w_gate_up.shape
    top = chosen.shape[1]
    _need(two == 2 and w_gate_up.is_contiguous() and h.stride(1) == 1 and h.shape[1] == width and h.dtype == w_gate_up.dtype == act.dtype
          and act.is_contiguous() and tuple(act.shape[1:]) == (top, ff) and act.shape[0] >= n_rows, "moe_gate_up: bad operands")
    _need(h.dtype == torch.float32 or (w_gate_up.data_ptr() % 16 == 0), "moe_gate_up: weights must be 16-byte aligned")
    code = _fn("moe", "tw_moe_gate_up")(_ptr(act), _ptr(h), c_int(h.stride(0)), _ptr(w_gate_up), _ptr(chosen), c_int(n_rows), c_int(width),
                                        c_int(ff), c_int(experts), c_int(top), c_int(glu), c_float(limit), c_float(alpha),
                                        c_int(dtype_code(h.dtype)), _stream())
    _check(code, "moe_gate_up")


def moe_up(act: torch.Tensor, h: torch.Tensor, w_up: torch.Tensor, chosen: torch.Tensor, n_rows: int, activation: int) -> None:
    """act[row, j] = f(Wu_e h[row]) for the j-th chosen expert e of the row: experts without a gate, ``w_up`` [experts, ff,
    width], f one of ``ACTIVATIONS``."""
    _cuda(act, h, w_up, chosen)
    experts, ff, width = w_up.shape
    top = chosen.shape[1]
    _need(w_up.is_contiguous() and h.stride(1) == 1 and h.shape[1] == width and h.dtype == w_up.dtype == act.dtype
          and act.is_contiguous() and tuple(act.shape[1:]) == (top, ff) and act.shape[0] >= n_rows, "moe_up: bad operands")
    _need(h.dtype == torch.float32 or (w_up.data_ptr() % 16 == 0), "moe_up: weights must be 16-byte aligned")
    code = _fn("moe", "tw_moe_up")(_ptr(act), _ptr(h), c_int(h.stride(0)), _ptr(w_up), _ptr(chosen), c_int(n_rows), c_int(width),
                                   c_int(ff), c_int(experts), c_int(top), c_int(activation), c_int(dtype_code(h.dtype)), _stream())
    _check(code, "moe_up")


def glu_rows(out: torch.Tensor, gate_up: torch.Tensor, n_rows: int, glu: int, limit: float = 0.0, alpha: float = 1.0) -> None:
    """out[n, i] = glu(gate_up[n, i], gate_up[n, I + i]) over rows [all gates | all ups] (see ``moe_gate_up``)."""
    _cuda(out, gate_up)
    inter = out.shape[1]
    _need(gate_up.shape[1] == 2 * inter and gate_up.is_contiguous() and out.is_contiguous() and gate_up.dtype == out.dtype
          and min(out.shape[0], gate_up.shape[0]) >= n_rows, "glu_rows: gate_up must be contiguous [n, 2I] of the output type")
    code = _fn("moe", "tw_glu_rows")(_ptr(out), _ptr(gate_up), c_int(n_rows), c_int(inter), c_int(glu), c_float(limit),
                                     c_float(alpha), c_int(dtype_code(out.dtype)), _stream())
    _check(code, "glu_rows")


def moe_down(out: torch.Tensor, act: torch.Tensor, w_down: torch.Tensor, chosen: torch.Tensor, weight: torch.Tensor,
             shared: torch.Tensor | None, shared_gate: torch.Tensor | None, n_rows: int,
             h: torch.Tensor | None = None, identity: int = 0) -> None:
    """out[row] = sum_j weight[row, j] * Wd_e act[row, j]  (+ shared_gate[row] * shared[row]); ``w_down`` is
    [experts, width, ff].  A chosen index in experts .. experts + ``identity`` - 1 adds weight * ``h[row]`` instead."""
    _cuda(out, act, w_down, chosen, weight, shared, shared_gate, h)
    _need(identity == 0 or (h is not None and h.stride(1) == 1 and h.dtype == out.dtype and h.shape[1] == out.shape[1]),
          "moe_down: identity experts need the rows themselves")
    experts, width, ff = w_down.shape
    top = chosen.shape[1]
    _need(w_down.is_contiguous() and act.is_contiguous() and tuple(act.shape[1:]) == (top, ff) and out.is_contiguous()
          and out.shape[1] == width and out.dtype == act.dtype == w_down.dtype, "moe_down: bad operands")
    _need(shared is None or (shared.is_contiguous() and shared.dtype == out.dtype and shared.shape[1] == width), "moe_down: bad shared rows")
    code = _fn("moe", "tw_moe_down")(_ptr(out), _ptr(act), _ptr(w_down), _ptr(chosen), _ptr(weight), _ptr(shared), _ptr(shared_gate),
                                     c_int(n_rows), c_int(width), c_int(ff), c_int(experts), c_int(top), _ptr(h),
                                     c_int(0 if h is None else h.stride(0)), c_int(identity), c_int(dtype_code(out.dtype)), _stream())
    _check(code, "moe_down")


def scaled_accumulate(acc: torch.Tensor, out: torch.Tensor | None, x: torch.Tensor, scale: float, first: bool) -> None:
    """acc = (0 if first else acc) + scale * x in fp32; ``out`` (may be None) receives the new sum in x's type."""
    _cuda(acc, out, x)
    _need(acc.dtype == torch.float32 and acc.is_contiguous() and x.is_contiguous() and acc.numel() == x.numel()
          and (out is None or (out.is_contiguous() and out.dtype == x.dtype and out.numel() == x.numel())),
          "scaled_accumulate: contiguous operands of one size, an fp32 sum")
    code = _fn("elementwise", "tw_scaled_accumulate")(_ptr(acc), _ptr(out), _ptr(x), c_float(scale), c_int(1 if first else 0),
                                                      ctypes.c_longlong(x.numel()), c_int(dtype_code(x.dtype)), _stream())
    _check(code, "scaled_accumulate")


def moe_sort(order: torch.Tensor, place: torch.Tensor, ends: torch.Tensor, chosen: torch.Tensor, n_rows: int) -> None:
    """Sort the (row, chosen expert) pairs of ``chosen[:n_rows]`` by expert: ``order[i]`` = the pair at sorted place
    i, ``place[pair]`` = its place, ``ends[e]`` = one past expert e's last place (all int32)."""
    _cuda(order, place, ends, chosen)
    top = chosen.shape[1]
    pairs = n_rows * top
    _need(all(t.dtype == torch.int32 and t.is_contiguous() for t in (order, place, ends, chosen)) and order.numel() >= pairs
          and place.numel() >= pairs, "moe_sort: int32 operands, one place per pair")
    code = _fn("moe", "tw_moe_sort")(_ptr(order), _ptr(place), _ptr(ends), _ptr(chosen), c_int(pairs), c_int(ends.numel()), _stream())
    _check(code, "moe_sort")


def moe_gather(xs: torch.Tensor, h: torch.Tensor, order: torch.Tensor, pairs: int, top: int) -> None:
    """xs[i] = h[order[i] // top]: every pair's input row, in sorted order."""
    _cuda(xs, h, order)
    _need(xs.is_contiguous() and xs.dtype == h.dtype and h.stride(1) == 1 and xs.shape[1] == h.shape[1] and xs.shape[0] >= pairs,
          "moe_gather: bad operands")
    code = _fn("moe", "tw_moe_gather")(_ptr(xs), _ptr(h), c_int(h.stride(0)), _ptr(order), c_int(pairs), c_int(top),
                                       c_int(h.shape[1]), c_int(dtype_code(h.dtype)), _stream())
    _check(code, "moe_gather")


def moe_combine(out: torch.Tensor, ys: torch.Tensor, place: torch.Tensor, weight: torch.Tensor, shared: torch.Tensor | None,
                shared_gate: torch.Tensor | None, n_rows: int, chosen: torch.Tensor | None = None, h: torch.Tensor | None = None,
                experts: int = 0, identity: int = 0) -> None:
    """out[row] = sum_j weight[row, j] * ys[place[row * top + j]]  (+ shared_gate[row] * shared[row]).  With
    ``identity`` a pair without a place whose chosen index lies in experts .. experts + identity - 1 adds
    weight * ``h[row]``."""
    _cuda(out, ys, place, weight, shared, shared_gate, chosen, h)
    _need(identity == 0 or (h is not None and chosen is not None and h.stride(1) == 1 and h.dtype == out.dtype
                            and h.shape[1] == out.shape[1] and chosen.dtype == torch.int32 and chosen.is_contiguous()),
          "moe_combine: identity experts need the chosen indices and the rows themselves")
    top, width = weight.shape[1], out.shape[1]
    _need(out.is_contiguous() and ys.is_contiguous() and ys.dtype == out.dtype and ys.shape[1] == width and weight.is_contiguous()
          and weight.dtype == torch.float32 and place.dtype == torch.int32, "moe_combine: bad operands")
    _need(shared is None or (shared.is_contiguous() and shared.dtype == out.dtype and shared.shape[1] == width), "moe_combine: bad shared rows")
    code = _fn("moe", "tw_moe_combine")(_ptr(out), _ptr(ys), _ptr(place), _ptr(weight), _ptr(shared), _ptr(shared_gate),
                                        c_int(n_rows), c_int(top), c_int(width), _ptr(chosen), _ptr(h),
                                        c_int(0 if h is None else h.stride(0)), c_int(experts), c_int(identity),
                                        c_int(dtype_code(out.dtype)), _stream())
    _check(code, "moe_combine")


def add_row_vector(resid: torch.Tensor, vec: torch.Tensor, n_rows: int) -> None:
    """resid[:n_rows] += vec: a learned fp32 vector added to every row of the fp32 residual stream."""
    _cuda(resid, vec)
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and vec.dtype == torch.float32 and vec.is_contiguous()
          and vec.numel() == resid.shape[1] and resid.shape[0] >= n_rows, "add_row_vector: fp32 [rows, width] and fp32 [width]")
    code = _fn("elementwise", "tw_add_row_vector")(_ptr(resid), _ptr(vec), c_int(n_rows), c_int(resid.shape[1]), _stream())
    _check(code, "add_row_vector")


def add_delta(resid: torch.Tensor, delta, n_rows: int) -> None:
    """resid[:n_rows] += delta in fp32; ``delta`` is a tensor [rows, width] (bfloat16 or fp32) or a ``SplitSum``."""
    width = resid.shape[1]
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and resid.shape[0] >= n_rows, "add_delta: the residual stream must be contiguous fp32")
    if isinstance(delta, SplitSum):
        slices = delta.slices
        _cuda(resid, slices)
        _need(slices.dtype == torch.float32 and slices.shape[2] == width and slices[0].is_contiguous() and slices.shape[1] >= n_rows,
              "add_delta: split sum must be fp32 [slices, rows, width]")
        code = _fn("elementwise", "tw_add_delta")(_ptr(resid), _ptr(None), _ptr(slices), c_int(slices.shape[0]),
                                                  ctypes.c_longlong(slices.stride(0)), ctypes.c_longlong(n_rows * width), c_int(F32), _stream())
    else:
        _cuda(resid, delta)
        _need(delta.is_contiguous() and delta.shape[1] == width and delta.shape[0] >= n_rows, "add_delta: delta must be contiguous [rows, width]")
        code = _fn("elementwise", "tw_add_delta")(_ptr(resid), _ptr(delta), _ptr(None), c_int(0), ctypes.c_longlong(0),
                                                  ctypes.c_longlong(n_rows * width), c_int(dtype_code(delta.dtype)), _stream())
    _check(code, "add_delta")


def normed_accumulate(acc: torch.Tensor, out: torch.Tensor | None, x: torch.Tensor, weight: torch.Tensor, eps: float, scale: float,
                      first: bool, n_rows: int) -> None:
    """acc[r] = (0 if first else acc[r]) + scale * x[r] / sqrt(mean(x[r]^2) + eps) * weight, row by row in fp32; ``out``
    (may be None) receives the new sum in x's type."""
    _cuda(acc, out, x, weight)
    width = x.shape[1]
    _need(acc.dtype == torch.float32 and acc.is_contiguous() and x.is_contiguous() and acc.shape[1] == width
          and min(acc.shape[0], x.shape[0]) >= n_rows and weight.dtype == torch.float32 and weight.is_contiguous() and weight.numel() == width
          and (out is None or (out.dtype == x.dtype and out.is_contiguous() and out.shape[1] == width and out.shape[0] >= n_rows)),
          "normed_accumulate: fp32 sum, rows of one type and shape, an fp32 weight of their width")
    code = _fn("elementwise", "tw_normed_accumulate")(_ptr(acc), _ptr(out), _ptr(x), _ptr(weight), c_float(eps), c_float(scale),
                                                      c_int(1 if first else 0), c_int(n_rows), c_int(width), c_int(dtype_code(x.dtype)), _stream())
    _check(code, "normed_accumulate")


WEIGHTED_SUM_MAX_MEMBERS = 4


def weighted_sum_rows(out: torch.Tensor, members: list[torch.Tensor], scales: list[float], weights: torch.Tensor | None,
                      eps: float, n_rows: int) -> None:
    """out[r] = sum_m scales[m] * members[m][r], or with ``weights`` ([members, width] fp32) the same over rows that are
    first divided by their root mean square (``eps`` inside the root) and multiplied by ``weights[m]``; fp32 statistics
    and sum, members added in their order, one rounding.  The members lie in buffers of their own."""
    _cuda(out, weights, *members)
    k, width = len(members), out.shape[1]
    _need(1 <= k <= WEIGHTED_SUM_MAX_MEMBERS and len(scales) == k, f"weighted_sum_rows: 1 to {WEIGHTED_SUM_MAX_MEMBERS} members, a scale each")
    _need(out.is_contiguous() and out.shape[0] >= n_rows
          and all(x.dtype == out.dtype and x.is_contiguous() and x.shape[1] == width and x.shape[0] >= n_rows
                  and x.data_ptr() != out.data_ptr() for x in members),
          "weighted_sum_rows: rows of one type and width, contiguous, none of them the result")
    _need(weights is None or (weights.dtype == torch.float32 and weights.is_contiguous() and tuple(weights.shape) == (k, width)),
          "weighted_sum_rows: the weights must be fp32 [members, width]")
    xs = [_ptr(x) for x in members] + [_ptr(None)] * (WEIGHTED_SUM_MAX_MEMBERS - k)
    sc = [c_float(float(v)) for v in scales] + [c_float(0.0)] * (WEIGHTED_SUM_MAX_MEMBERS - k)
    code = _fn("elementwise", "tw_weighted_sum_rows")(_ptr(out), *xs, *sc, _ptr(weights), c_float(float(eps or 0.0)), c_int(k),
                                                      c_int(n_rows), c_int(width), c_int(dtype_code(out.dtype)), _stream())
    _check(code, "weighted_sum_rows")


SHORT_CONV_MAX_TAPS = 17


def short_conv(out: torch.Tensor, x: torch.Tensor, w: torch.Tensor, state: torch.Tensor, state_offset: int,
               seq_of_token: torch.Tensor, seq_slot: torch.Tensor, seq_q_start: torch.Tensor, n_rows: int,
               unit_heads: int = 0, unit_dim: int = 0, scaled_heads: int = 0, head_scale: float = 1.0, unit_eps: float = 0.0,
               move_single: torch.Tensor | None = None, bias: torch.Tensor | None = None) -> None:
    """out[t, c] = silu([bias[c] +] sum_j w[c, j] x[t - (taps - 1) + j, c]) as fp32 or bf16 rows [rows, channels]: a causal convolution over the
    rows of each request, per channel (the last tap is the row's own).  The taps - 1 rows before a request's first row of
    this step are read from its state (fp32, [channels, taps - 1] at ``state_offset``; zeros at a request's start).  The
    first ``unit_heads`` heads of ``unit_dim`` channels are then scaled to x / sqrt(sum x^2 + unit_eps), the first
    ``scaled_heads`` of those also by ``head_scale``.  ``short_conv_state`` moves the state on afterwards; with
    ``move_single`` (the requests' row counts of this step, int32) the kernel itself moves on the state of every request
    that brings one row, and ``short_conv_state(..., skip_single=True)`` is needed only for the others."""
    _cuda(out, x, w, state, seq_of_token, seq_slot, seq_q_start, move_single, bias)
    _need(bias is None or (bias.dtype == torch.float32 and bias.is_contiguous() and bias.numel() == w.shape[0]), "short_conv: the bias must be fp32 [channels]")
    _need(move_single is None or move_single.dtype == torch.int32, "short_conv: the row counts must be int32")
    channels, taps = w.shape
    _need(out.dtype in (torch.float32, x.dtype) and out.is_contiguous() and out.shape[1] == channels and out.shape[0] >= n_rows,
          "short_conv: the result must be contiguous [rows, channels], in fp32 or x's type")
    _need(x.stride(1) == 1 and x.shape[1] >= channels and x.shape[0] >= n_rows, "short_conv: bad input rows")
    _need(w.dtype == torch.float32 and 1 <= taps <= SHORT_CONV_MAX_TAPS, "short_conv: taps must be fp32 [channels, 1..17]")
    _need(state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1
          and state_offset + channels * (taps - 1) <= state.shape[1], "short_conv: the state must be fp32 [slots, numel] with room for the taps")
    _need(0 <= scaled_heads <= unit_heads and unit_heads * unit_dim <= channels, "short_conv: the unit heads exceed the channels")
    code = _fn("recurrent", "tw_short_conv")(
        _ptr(out), _ptr(x), c_int(x.stride(0)), _ptr(w), c_int(w.stride(0)), c_int(w.stride(1)), _ptr(bias), c_int(taps), _ptr(state), ctypes.c_longlong(state.stride(0)),
        ctypes.c_longlong(state_offset), _ptr(seq_of_token), _ptr(seq_slot), _ptr(seq_q_start), _ptr(move_single),
        c_int(0 if move_single is None else 1), c_int(n_rows), c_int(channels),
        c_int(unit_heads), c_int(unit_dim), c_int(scaled_heads), c_float(head_scale), c_float(unit_eps), c_int(dtype_code(x.dtype)),
        c_int(dtype_code(out.dtype)), _stream())
    _check(code, "short_conv")


def short_conv_state(x: torch.Tensor, taps: int, channels: int, state: torch.Tensor, state_offset: int, seq_slot: torch.Tensor,
                     seq_q_start: torch.Tensor, seq_q_len: torch.Tensor, n_seqs: int, skip_single: bool = False) -> None:
    """After ``short_conv``: every request's state keeps the last ``taps - 1`` inputs (older ones stay where the step
    brought fewer rows than that).  ``skip_single``: requests with one row are left as they are."""
    _cuda(x, state, seq_slot, seq_q_start, seq_q_len)
    _need(x.stride(1) == 1 and x.shape[1] >= channels and 1 <= taps <= SHORT_CONV_MAX_TAPS, "short_conv_state: bad input rows or taps")
    _need(state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1
          and state_offset + channels * (taps - 1) <= state.shape[1], "short_conv_state: the state must be fp32 [slots, numel] with room for the taps")
    code = _fn("recurrent", "tw_short_conv_state")(
        _ptr(x), c_int(x.stride(0)), c_int(taps), _ptr(state), ctypes.c_longlong(state.stride(0)), ctypes.c_longlong(state_offset),
        _ptr(seq_slot), _ptr(seq_q_start), _ptr(seq_q_len), c_int(n_seqs), c_int(channels), c_int(1 if skip_single else 0),
        c_int(dtype_code(x.dtype)), _stream())
    _check(code, "short_conv_state")

"""Thin typed wrappers over the C ABI: torch tensors own the device memory, every call is one or two
kernel launches on torch's current CUDA stream.  No arithmetic happens in Python or in torch here."""
import ctypes
import functools
import math

import torch

from . import _lib
from ._lib import BF16, BFP4, BFP8, FP32, check, lib

_TORCH = {"bf16": torch.bfloat16, "fp32": torch.float32, "int32": torch.int32}
_CODES = {torch.bfloat16: BF16, torch.float32: FP32, torch.int32: _lib.INT32}

KERNELS = [0]  # kernels of this library launched so far by this process (every wrapper below counts its own)


def count(n=1):
    KERNELS[0] += n


def _stream():
    return torch.cuda.current_stream().cuda_stream


def _ptr(t):
    return None if t is None else t.data_ptr()


class Packed:
    """A batch of block-float matrices [batch, K, N] on the device (include/ferrite_b200.h says how the bytes lie)."""

    def __init__(self, fmt, batch, K, N, data):
        self.fmt, self.batch, self.K, self.N, self.data = fmt, batch, K, N, data

    @property
    def code(self):
        return _lib.DTYPES[self.fmt]

    @property
    def matrix_bytes(self):
        return lib().fb_packed_bytes(self.code, self.K, self.N)

    def matrix(self, e):
        """Matrix e of the batch, in place."""
        n = self.matrix_bytes
        return Packed(self.fmt, 1, self.K, self.N, self.data[e * n:(e + 1) * n])


def quantize(x, fmt):
    """bf16 [K, N] or [batch, K, N] -> Packed (Tensor.cast to a block float, ferrite/tensor.py:315-320)."""
    assert x.dtype == torch.bfloat16 and x.is_cuda and x.is_contiguous(), "a contiguous bf16 CUDA tensor"
    batch, K, N = (1, *x.shape) if x.dim() == 2 else x.shape
    n = lib().fb_packed_bytes(_lib.DTYPES[fmt], K, N)
    assert n, f"{tuple(x.shape)} to {fmt}: columns in runs of 16"
    data = torch.empty(batch * n, dtype=torch.uint8, device=x.device)
    check(lib().fb_quantize(_lib.DTYPES[fmt], x.data_ptr(), batch, K, N, data.data_ptr(), _stream()))
    count()
    return Packed(fmt, batch, K, N, data)


def dequantize(p):
    """Packed -> bf16 [batch, K, N]: the values, each exactly a bf16."""
    out = torch.empty(p.batch, p.K, p.N, dtype=torch.bfloat16, device=p.data.device)
    check(lib().fb_dequantize(p.code, p.data.data_ptr(), p.batch, p.K, p.N, out.data_ptr(), _stream()))
    return out


def unpack_fields(p):
    """Packed -> (top [batch,K,N/16], sign [batch,K,N], mag [batch,K,N]) uint8."""
    dev = p.data.device
    top = torch.empty(p.batch, p.K, p.N // 16, dtype=torch.uint8, device=dev)
    sign = torch.empty(p.batch, p.K, p.N, dtype=torch.uint8, device=dev)
    mag = torch.empty_like(sign)
    check(lib().fb_unpack_fields(p.code, p.data.data_ptr(), p.batch, p.K, p.N, top.data_ptr(), sign.data_ptr(), mag.data_ptr(), _stream()))
    return top, sign, mag


_WORKSPACES = {}
_RETIRED = []  # scratch buffers a larger one has replaced: a recorded CUDA graph may still hold their addresses


def _scratch(table, device, nbytes, least):
    """The device's buffer of one kind of scratch: zeroed when made, replaced by a larger one when a call needs more.
    The one it replaces is kept alive for good: a step recorded by `jit` replays kernels that were given its address."""
    have = table.get(device)
    if have is None or have.numel() < nbytes:
        if have is not None:
            _RETIRED.append(have)
        have = table[device] = torch.zeros(max(nbytes, least), dtype=torch.uint8, device=device)
    return have


def linear_workspace(device, nbytes):
    """The device's scratch buffer for fb_linear (the normalised activations of a fused RMSNorm, the partial tiles and
    arrival counters of tiles shared by several CTAs): one per device, zeroed when made (the counters start at 0 and
    every call leaves them 0).  Calls on one stream run in order, so they can share it."""
    return _scratch(_WORKSPACES, device, nbytes, 64 << 20) if nbytes else None


def linear(x, w, out=None, out_dtype="bf16", norm_w=None, eps=1e-5, epilogue="none", residual=None, workspace=None):
    """x [M, K] bf16 @ w (Packed, one matrix) with the fused RMSNorm prologue / SwiGLU or residual epilogue."""
    assert x.dtype == torch.bfloat16 and x.dim() == 2 and x.stride(1) == 1 and w.batch == 1 and x.shape[1] == w.K, \
        f"{tuple(x.shape)} @ [{w.K}, {w.N}]"
    M, K = x.shape
    epi = {"none": _lib.EPI_NONE, "swiglu": _lib.EPI_SWIGLU, "residual": _lib.EPI_RESIDUAL}[epilogue]
    cols = w.N // 2 if epilogue == "swiglu" else w.N
    if out is None:
        out = torch.empty(M, cols, dtype=_TORCH[out_dtype], device=x.device)
    assert out.shape == (M, cols) and out.stride(1) == 1 and out.dtype == _TORCH[out_dtype]
    if workspace is None:
        workspace = linear_workspace(x.device, lib().fb_linear_workspace_bytes(M, K, w.N))
    check(lib().fb_linear(w.code, x.data_ptr(), M, K, x.stride(0), w.data.data_ptr(), w.N, out.data_ptr(), _lib.DTYPES[out_dtype],
                          out.stride(0), _ptr(norm_w), eps, epi, _ptr(residual), residual.stride(0) if residual is not None else 0,
                          _ptr(workspace), workspace.numel() if workspace is not None else 0, _stream()))
    count(1 if M <= 1 else -(-M // 128) * (2 if norm_w is not None else 1))  # the GEMV, or GEMM passes (+ the norm's)
    return out


def chain_parts(w, M, epilogue="none"):
    """How many parts the sums of squares of fb_linear_chained's result come in for this shape; 0: it cannot hand a norm on."""
    epi = {"none": _lib.EPI_NONE, "swiglu": _lib.EPI_SWIGLU, "residual": _lib.EPI_RESIDUAL}[epilogue]
    return lib().fb_linear_chain_parts(w.code, M, w.K, w.N, epi)


def linear_chained(x, w, out=None, out_dtype="bf16", eps=1e-5, epilogue="none", residual=None, norm_in=None, next_norm_w=None):
    """fb_linear_chained: x @ w with an RMSNorm taken over from the matmul before (norm_in = (sumsq, parts): x is that
    matmul's xn) and / or handed on to the one after (next_norm_w: returns (out, xn, sumsq, parts) instead of out)."""
    assert x.dtype == torch.bfloat16 and x.dim() == 2 and x.stride(1) == 1 and w.batch == 1 and x.shape[1] == w.K
    M = x.shape[0]
    epi = {"none": _lib.EPI_NONE, "swiglu": _lib.EPI_SWIGLU, "residual": _lib.EPI_RESIDUAL}[epilogue]
    cols = w.N // 2 if epilogue == "swiglu" else w.N
    if out is None:
        out = torch.empty(M, cols, dtype=_TORCH[out_dtype], device=x.device)
    xn = sumsq = None
    parts = 0
    if next_norm_w is not None:
        parts = chain_parts(w, M, epilogue)
        assert parts, "this shape cannot hand a norm on"
        xn = torch.empty(M, w.N, dtype=torch.bfloat16, device=x.device)
        sumsq = torch.empty(parts, M, dtype=torch.float32, device=x.device)
    check(lib().fb_linear_chained(w.code, x.data_ptr(), M, w.K, x.stride(0), w.data.data_ptr(), w.N, out.data_ptr(), _lib.DTYPES[out_dtype], out.stride(0),
                                  eps, epi, _ptr(residual), residual.stride(0) if residual is not None else 0,
                                  _ptr(norm_in[0]) if norm_in else None, norm_in[1] if norm_in else 0, _ptr(next_norm_w), _ptr(xn),
                                  xn.stride(0) if xn is not None else 0, _ptr(sumsq), None, 0, _stream()))
    count()
    return (out, xn, sumsq, parts) if next_norm_w is not None else out


def gather_rows(table, ids, out=None):
    """table[ids] for a 2-D table and an int32 vector of ids on the device (Tensor.gather)."""
    assert table.dim() == 2 and table.is_contiguous() and ids.dtype == torch.int32 and ids.dim() == 1
    if out is None:
        out = torch.empty(ids.numel(), table.shape[1], dtype=table.dtype, device=table.device)
    check(lib().fb_gather_rows(table.data_ptr(), table.shape[0], table.shape[1] * table.element_size(), ids.data_ptr(), ids.numel(),
                               out.data_ptr(), _stream()))
    count()
    return out


def rope_kv_write(qkv, cos, sin, places, rows, cache, H, KV, hd, q_out=None, qk_norm=None, eps=1e-5):
    """RoPE (and Qwen3's q/k norm) on a fused qkv [T, (H+2KV)*hd]; q -> q_out [T, H*hd], k and v into cache
    [2*KV, cache_rows, hd] at rows (a bf16 tensor, or a Packed block-float batch of 2*KV matrices [cache_rows, hd])."""
    T = qkv.shape[0]
    assert qkv.dtype == torch.bfloat16 and qkv.shape[1] == (H + 2 * KV) * hd and qkv.stride(1) == 1
    if isinstance(cache, Packed):
        assert cache.batch == 2 * KV and cache.N == hd and places.dtype == torch.int32 and rows.dtype == torch.int32
        if q_out is None:
            q_out = torch.empty(T, H * hd, dtype=torch.bfloat16, device=qkv.device)
        check(lib().fb_rope_kv_write_packed(cache.code, qkv.data_ptr(), T, qkv.stride(0), H, KV, hd, cos.data_ptr(), sin.data_ptr(), cos.shape[-1],
                                            cos.shape[0], places.data_ptr(), rows.data_ptr(), _ptr(qk_norm), eps, q_out.data_ptr(), q_out.stride(0),
                                            cache.data.data_ptr(), cache.K, _stream()))
        count()
        return q_out
    assert cache.dtype == torch.bfloat16 and cache.shape[0] == 2 * KV and cache.shape[2] == hd and cache.stride(2) == 1 and cache.stride(1) == hd
    assert places.dtype == torch.int32 and rows.dtype == torch.int32 and places.numel() == T and rows.numel() == T
    assert cos.shape == sin.shape and cos.is_contiguous() and sin.is_contiguous() and cos.dtype == torch.bfloat16
    if q_out is None:
        q_out = torch.empty(T, H * hd, dtype=torch.bfloat16, device=qkv.device)
    check(lib().fb_rope_kv_write(qkv.data_ptr(), T, qkv.stride(0), H, KV, hd, cos.data_ptr(), sin.data_ptr(), cos.shape[-1], cos.shape[0], places.data_ptr(),
                                 rows.data_ptr(), _ptr(qk_norm), eps, q_out.data_ptr(), q_out.stride(0), cache.data_ptr(), cache.shape[1], cache.stride(0), _stream()))
    count()
    return q_out


_ATT_WS = {}


def decode_attention(q, cache, base, place, H, KV, hd, max_keys, window=0, out=None):
    """One token per sequence: token t attends cache rows base[t] .. base[t] + place[t] of its kv head."""
    T = q.shape[0]
    packed = isinstance(cache, Packed)  # a block-float cache: sequences start at multiples of 64 rows (base)
    assert q.dtype == torch.bfloat16 and q.shape[1] == H * hd and q.stride(1) == 1
    assert (cache.batch == 2 * KV and cache.N == hd) if packed else (cache.stride(2) == 1 and cache.stride(1) == hd)
    assert base.dtype == torch.int32 and place.dtype == torch.int32 and base.numel() == T and place.numel() == T
    if out is None:
        out = torch.empty(T, H * hd, dtype=torch.bfloat16, device=q.device)
    need = lib().fb_decode_attention_workspace_bytes(T, H, KV, hd, max_keys)
    ws = attention_workspace(q.device, need)
    if packed:
        check(lib().fb_decode_attention_packed(cache.code, q.data_ptr(), T, q.stride(0), H, KV, hd, cache.data.data_ptr(), cache.K, base.data_ptr(),
                                               place.data_ptr(), max_keys, window, out.data_ptr(), out.stride(0), _ptr(ws) if need else None,
                                               ws.numel() if need else 0, _stream()))
    else:
        check(lib().fb_decode_attention(q.data_ptr(), T, q.stride(0), H, KV, hd, cache.data_ptr(), cache.shape[1], cache.stride(0), base.data_ptr(),
                                        place.data_ptr(), max_keys, window, out.data_ptr(), out.stride(0), _ptr(ws) if need else None,
                                        ws.numel() if need else 0, _stream()))
    count(2 if need else 1)  # the attention kernel, and the merge of its key splits
    return out


def prefill_attention(q, cache, first_row, places, H, KV, hd, max_keys, window=0, out=None):
    """A chunk of one sequence's prompt: token t (at places[t]) attends the cache rows first_row .. first_row + places[t]
    of its kv head; 16 tokens of a query head share every key row read."""
    T = q.shape[0]
    packed = isinstance(cache, Packed)
    assert q.dtype == torch.bfloat16 and q.shape[1] == H * hd and q.stride(1) == 1 and places.dtype == torch.int32 and places.numel() == T
    assert (cache.batch == 2 * KV and cache.N == hd) if packed else (cache.stride(2) == 1 and cache.stride(1) == hd)
    if out is None:
        out = torch.empty(T, H * hd, dtype=torch.bfloat16, device=q.device)
    need = lib().fb_prefill_attention_workspace_bytes(T, H, hd, max_keys)
    ws = attention_workspace(q.device, need)
    check(lib().fb_prefill_attention(cache.code if packed else BF16, q.data_ptr(), T, q.stride(0), H, KV, hd, cache.data.data_ptr() if packed else cache.data_ptr(),
                                     cache.K if packed else cache.shape[1], 0 if packed else cache.stride(0), first_row, places.data_ptr(), max_keys, window,
                                     out.data_ptr(), out.stride(0), _ptr(ws) if need else None, ws.numel() if need else 0, _stream()))
    count(2 if need else 1)
    return out


def rmsnorm(x, w, eps=1e-5, out=None):
    assert x.dtype == torch.bfloat16 and x.dim() == 2 and x.stride(1) == 1 and w.numel() == x.shape[1]
    if out is None:
        out = torch.empty_like(x)
    check(lib().fb_rmsnorm(x.data_ptr(), x.shape[0], x.shape[1], x.stride(0), w.data_ptr(), eps, out.data_ptr(), out.stride(0), _stream()))
    count()
    return out


def argmax(logits, out=None, values=None):
    """Each row's first largest fp32 logit's column (int32); values: an fp32 vector that receives the maxima."""
    assert logits.dtype == torch.float32 and logits.dim() == 2 and logits.stride(1) == 1
    if out is None:
        out = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
    check(lib().fb_argmax(logits.data_ptr(), logits.shape[0], logits.shape[1], logits.stride(0), out.data_ptr(), _ptr(values), _stream()))
    count()
    return out


def attention_workspace(device, nbytes):
    """The device's scratch for the attention kernels' key splits (a larger one replaces it when a call needs more;
    the replaced one stays alive for the recorded steps that hold its address)."""
    return _scratch(_ATT_WS, device, nbytes, 16 << 20) if nbytes else None


def linear_indexed(x, w, index, out, sum_slots=False, x_slot_rows=0, out_slot_stride=0, M=None, out_dtype="bf16", norm_w=None, eps=1e-5,
                   epilogue="none", residual=None, row_scale=None):
    """A mixture of experts' matmul: x [M, K] (or n_slots of them, or [M, n_slots * K] with sum_slots) by the matrices
    of the batch w (Packed) that index (int32 [n_slots], on the device) picks; see fb_linear_indexed."""
    M = x.shape[0] if M is None else M
    n_slots = index.numel()
    assert x.dtype == torch.bfloat16 and x.stride(1) == 1 and index.dtype == torch.int32 and index.is_contiguous()
    epi = {"none": _lib.EPI_NONE, "swiglu": _lib.EPI_SWIGLU, "residual": _lib.EPI_RESIDUAL}[epilogue]
    ws = linear_workspace(x.device, lib().fb_linear_workspace_bytes(max(M, 5), w.K, w.N)) if norm_w is not None else None
    check(lib().fb_linear_indexed(w.code, x.data_ptr(), M, w.K, x.stride(0), x_slot_rows, w.data.data_ptr(), w.N, w.batch, index.data_ptr(), n_slots,
                                  int(sum_slots), out.data_ptr(), _lib.DTYPES[out_dtype], out.stride(-2), out_slot_stride, _ptr(norm_w), eps, epi,
                                  _ptr(residual), residual.stride(0) if residual is not None else 0, _ptr(row_scale), _ptr(ws),
                                  ws.numel() if ws is not None else 0, _stream()))
    count(2 if norm_w is not None else 1)
    return out


def latent_put(down, q_rank, kv_rank, rot, dims, q_norm, kv_norm, eps, freq, mag, places, rows, cache, q_out, heads=0, dim=0, q_turned=None):
    """The norms, the turn and the cache write after a joint down-projection (fb_latent_put); q_turned: [heads, T, rot]."""
    check(lib().fb_latent_put(_CODES[down.dtype], down.data_ptr(), down.shape[0], down.stride(0), q_rank, kv_rank, rot, dims, _ptr(q_norm), kv_norm.data_ptr(), eps,
                              freq.data_ptr(), mag, places.data_ptr(), rows.data_ptr(), _CODES[cache.dtype], _ptr(q_out), q_out.stride(0) if q_out is not None else 0,
                              heads, dim, _ptr(q_turned), q_turned.stride(1) if q_turned is not None else 0, q_turned.stride(0) if q_turned is not None else 0,
                              cache.data_ptr(), cache.shape[0], _stream()))
    count()


def rotate_pairs(x, rotation, places, out):
    """x [heads, T, width] -> out, the first columns of each head turned (fb_rotate_pairs)."""
    freq, dims, mag = rotation
    check(lib().fb_rotate_pairs(_CODES[x.dtype], x.data_ptr(), x.shape[1], x.shape[0], x.stride(1), x.stride(0), x.shape[2], dims, freq.data_ptr(), mag,
                                places.data_ptr(), out.data_ptr(), out.stride(1), out.stride(0), _stream()))
    count()
    return out


def latent_attention(q, cache, base, last, heads, rank, scale, sink, max_keys, chunk, row0=0, out=None, window=0):
    """q [T, heads * (rank + rot)] over cache [rows, rank + rot] (fb_latent_attention)."""
    T, rot = q.shape[0], cache.shape[1] - rank
    if out is None:
        out = torch.empty(T, heads * rank, dtype=q.dtype, device=q.device)
    assert cache.is_contiguous() and last.numel() == T and (base is None or base.numel() == T) and last.dtype == torch.int32
    code = _CODES[q.dtype]
    need = lib().fb_latent_attention_workspace_bytes(code, T, heads, rank, rot, max_keys, int(chunk), window)
    ws = attention_workspace(q.device, need)
    check(lib().fb_latent_attention(code, q.data_ptr(), T, q.stride(0), heads, rank, rot, cache.data_ptr(), cache.shape[0], _ptr(base), row0, last.data_ptr(), max_keys,
                                    int(chunk), window, scale, _ptr(sink), out.data_ptr(), out.stride(0), _ptr(ws) if need else None, ws.numel() if need else 0, _stream()))
    count(2 if need else 1)
    return out


def decay_scan(qkv, heads, dim, vdim, decay, places, dead, state, out):
    """Linear attention with decay over state [sequences, heads * dim, vdim] (fb_decay_scan)."""
    sequences = state.shape[0]
    assert state.stride(2) == 1 and state.stride(1) == vdim and places.dtype == torch.int32 and places.numel() == qkv.shape[0]
    check(lib().fb_decay_scan(_CODES[qkv.dtype], qkv.data_ptr(), qkv.stride(0), heads, dim, vdim, decay.data_ptr(), places.data_ptr(), dead, sequences,
                              qkv.shape[0] // sequences, state.data_ptr(), state.stride(0), out.data_ptr(), out.stride(0), _stream()))
    count()
    return out


def selective_scan(xbc, heads, groups, dim, vdim, step, step_bias, a_log, skip, places, dead, state, out):
    """A state space whose decay and step size are a token's own, over state [sequences, heads * dim, vdim] (fb_selective_scan)."""
    sequences = state.shape[0]
    assert state.stride(2) == 1 and state.stride(1) == vdim and places.dtype == torch.int32 and places.numel() == xbc.shape[0] and step.dtype == torch.float32 and step.stride(1) == 1
    check(lib().fb_selective_scan(_CODES[xbc.dtype], xbc.data_ptr(), xbc.stride(0), heads, groups, dim, vdim, step.data_ptr(), step.stride(0), step_bias.data_ptr(), a_log.data_ptr(), skip.data_ptr(),
                                  places.data_ptr(), dead, sequences, xbc.shape[0] // sequences, state.data_ptr(), state.stride(0), out.data_ptr(), out.stride(0), _stream()))
    count()
    return out


def short_conv(x, w, out, places, dead, state=None, bias=None, in_bias=None, silu=False):
    """A causal convolution over time of each column (fb_short_conv): w [taps, columns], state [sequences, >= taps - 1, columns]."""
    taps, cols = w.shape
    sequences = 1 if state is None else state.shape[0]
    assert x.shape[1] == out.shape[1] == cols and w.is_contiguous() and (state is None or (state.dtype == torch.float32 and state.shape[1] >= taps - 1 and state.shape[2] == state.stride(1) == cols and state.stride(2) == 1))
    c = _lib.Conv(cols, taps, w.data_ptr(), _ptr(bias), _ptr(in_bias), int(silu), places.data_ptr(), dead, sequences, x.shape[0] // sequences, _ptr(state), state.stride(0) if state is not None else 0)
    check(lib().fb_short_conv(ctypes.byref(c), _CODES[x.dtype], x.data_ptr(), x.stride(0), _CODES[out.dtype], out.data_ptr(), out.stride(0), _stream()))
    count()
    return out


def lru_scan(u, gates, y, out, lam, rate, blocks, places, dead, state, gate_bias=None, y_bias=None, scale=1.0):
    """A gated linear recurrence per column times the GELU of y (fb_lru_scan): state [sequences, 1, width]."""
    sequences, width = state.shape[0], u.shape[1]
    assert state.shape[2] == width and state.stride(2) == 1 and state.dtype == gates.dtype == torch.float32 and u.dtype == out.dtype and gates.shape[1] == 2 * width and lam.numel() == width
    l = _lib.Lru(width, blocks, lam.data_ptr(), rate, _ptr(gate_bias), _ptr(y_bias), scale, places.data_ptr(), dead, sequences, u.shape[0] // sequences, state.data_ptr(), state.stride(0))
    check(lib().fb_lru_scan(ctypes.byref(l), _CODES[u.dtype], u.data_ptr(), u.stride(0), gates.data_ptr(), gates.stride(0), _CODES[y.dtype], y.data_ptr(), y.stride(0), out.data_ptr(), out.stride(0),
                            _stream()))
    count()
    return out


def gated_rmsnorm(x, gate, w, eps, out, before=False, parts=1):
    """RMSNorm of x's rows in equal parts by w, times the sigmoid of gate (before: of x times its SiLU) (fb_gated_rmsnorm)."""
    check(lib().fb_gated_rmsnorm(x.data_ptr(), x.shape[0], x.shape[1], x.stride(0), _CODES[gate.dtype], gate.data_ptr(), gate.stride(0), int(before), w.data_ptr(), eps, parts,
                                 _CODES[out.dtype], out.data_ptr(), out.stride(0), _stream()))
    count()
    return out


def dense_supports(x, w, kind=_lib.DENSE_NONE):
    """Whether fb_dense takes x [batch, M, K] by w [batch, K, N], both bf16 views, w with each column's values together."""
    return x.dtype == w.dtype == torch.bfloat16 and x.stride(2) == 1 and w.stride(1) == 1 and bool(
        lib().fb_dense_supports(x.data_ptr(), x.stride(1), x.stride(0) if x.shape[0] > 1 else 0, w.data_ptr(), w.stride(2), w.stride(0) if w.shape[0] > 1 else 0,
                                w.shape[1], w.shape[2], kind))


def dense(x, w, out, settled=False, /, kind=_lib.DENSE_NONE, **extra):
    """x [batch, M, K] @ w [batch, K, N] into out [batch, M, columns] by fb_dense; extra: the fields of the epilogue's struct."""
    e = _lib.DenseEpilogue(kind=kind, **extra)
    batch = x.shape[0]
    assert out.stride(2) == 1 and out.shape[0] == batch == w.shape[0] and out.shape[1] == x.shape[1]
    check(lib().fb_dense(x.data_ptr(), x.shape[1], w.shape[1], x.stride(1), x.stride(0) if batch > 1 else 0, w.data_ptr(), w.shape[2], w.stride(2),
                         w.stride(0) if batch > 1 else 0, batch, out.data_ptr(), _CODES[out.dtype], out.stride(1), out.stride(0), ctypes.byref(e), int(settled), _stream()))
    count()
    return out


def embed(table, ids, places_table, places, out, scale=1.0):
    """out (fp32) = table[ids] * scale + places_table[places] (fb_embed)."""
    check(lib().fb_embed(_CODES[table.dtype], table.data_ptr(), table.shape[0], table.shape[1], ids.data_ptr(), _ptr(places_table), places_table.shape[0] if places_table is not None else 0,
                         _ptr(places), ids.numel(), scale, out.data_ptr(), _stream()))
    count()
    return out


def heads_put(qkv, heads, kv_heads, dim, vdim, rows, cache, q_out, bias=None, q_norm=None, k_norm=None, eps=0.0, first=None, first_bias=None, share=None,
              norm_all=False, keys_are_values=False, rotation=None, places=None, conv=None, state=None, dead=-1, temperature=(0.0, 1.0)):
    """Biases, convolution, norms, turn, values and the cache write after a joint projection of heads (fb_heads_put); cache [kv_heads,
    rows, dim + vdim]; rotation: (frequencies, columns that turn, factor); conv [taps, columns] and state [sequences, taps - 1, columns];
    temperature: (coefficient, places a step)."""
    freq, dims, mag = rotation or (None, 0, 1.0)
    h = _lib.Heads(heads, kv_heads, dim, vdim, _ptr(bias), _ptr(q_norm), _ptr(k_norm), eps, _ptr(first), first.stride(0) if first is not None else 0, _ptr(first_bias), _ptr(share),
                   int(norm_all), int(keys_are_values), dims, _ptr(freq) if dims else None, mag, _ptr(places), conv.shape[0] if conv is not None else 0, _ptr(conv), _ptr(state),
                   state.stride(0) if state is not None else 0, state.shape[0] if state is not None else 1, dead, *temperature)
    assert conv is None or (conv.is_contiguous() and state.dtype == conv.dtype == torch.float32 and state.shape[2] == state.stride(1) == conv.shape[1] and state.stride(2) == 1 and state.shape[1] >= conv.shape[0] - 1)
    assert cache.shape[0] == kv_heads and cache.shape[2] == dim + vdim and cache.stride(2) == 1 and cache.stride(1) == dim + vdim and q_out.dtype == cache.dtype
    check(lib().fb_heads_put(ctypes.byref(h), _CODES[qkv.dtype], qkv.data_ptr(), qkv.shape[0], qkv.stride(0), rows.data_ptr(), _CODES[cache.dtype], q_out.data_ptr(), q_out.stride(0),
                             cache.data_ptr(), cache.shape[1], cache.stride(0), _stream()))
    count()
    return q_out


def heads_attention(q, cache, base, last, heads, vdim, scale, max_keys, chunk, span=0, sink=None, gate=None, row0=0, out=None, window=0, softcap=0.0, key_bias=None,
                    out_scale=1.0):
    """q [T, heads * dim] over cache [kv_heads, rows, dim + vdim] (fb_heads_attention)."""
    T, dim = q.shape[0], cache.shape[2] - vdim
    assert q.shape[1] == heads * dim and q.dtype == cache.dtype and cache.stride(2) == 1 and cache.stride(1) == cache.shape[2]
    assert last.dtype == torch.int32 and last.numel() == T and (base is None or base.numel() == T)
    if out is None:
        out = torch.empty(T, heads * vdim, dtype=q.dtype, device=q.device)
    check(lib().fb_heads_attention(_CODES[q.dtype], q.data_ptr(), T, q.stride(0), heads, cache.shape[0], dim, vdim, cache.data_ptr(), cache.shape[1], cache.stride(0), _ptr(base), row0,
                                   last.data_ptr(), max_keys, int(chunk), span, window, scale, softcap, _ptr(sink), _ptr(key_bias), out_scale, _CODES[gate.dtype] if gate is not None else 0, _ptr(gate),
                                   gate.stride(0) if gate is not None else 0, out.data_ptr(), out.stride(0), _stream()))
    count()
    return out


class Routes:
    """Where a mixture's rows go (fb_route): tokens' weights, choices and slots [T, k], the tiles' experts, how many tiles are in
    use, and the sizes of all that (n: the experts that have rows); shared: every tile holds all the tokens."""

    def __init__(self, device, T, n, k, tile, shared):
        self.T, self.n, self.k, self.tile, self.shared = T, n, k, tile, shared
        self.tiles = lib().fb_route_tiles(T, n, k, tile, int(shared))
        i32 = lambda *shape: torch.empty(*shape, dtype=torch.int32, device=device)
        self.weights, self.ids, self.slots = torch.empty(T, k, dtype=torch.float32, device=device), i32(T, k), i32(T, k)
        self.tile_expert, self.live = i32(self.tiles, 3), i32(1)
        self.row_weights = None  # where weights go on the experts' inputs: each row's


@functools.lru_cache
def route_tile(T, n, k):
    """(rows of a tile, whether each tile holds all the tokens) for T tokens with k of n experts each: a few tokens are not
    sorted.  More: the height at which evenly drawn choices make for the least work, a tile costing what its weights' way
    through a CTA does (as much as 110 rows' products, measured) or its products."""
    if T <= 64:
        return -(-T // 16) * 16, True
    m = T * k / n
    spread = (m * (1 - k / n)) ** 0.5 + 1e-9
    above = lambda x: 0.5 * math.erfc((x - m) / (spread * 2 ** 0.5))  # how likely an expert has more than x rows
    work = lambda tile: sum(above(j * tile) for j in range(int((m + 5 * spread) / tile) + 2)) * max(110 + 0.1 * tile, tile)
    return min(range(32, 257, 16), key=work), False


SCORES = {False: 0, None: 0, True: 1, "softmax": 1, "sigmoid": 2}  # fb_router's scored


def route(logits, n, k, bias=None, scored=False, identity=0, scale=1.0, as_scored=False, on_input=False):
    """Router logits (fp32 [T, >= n]) to Routes; scored, identity, scale, as_scored: fb_router's; on_input: the weights by row, too."""
    T = logits.shape[0]
    tile, shared = route_tile(T, n, k)
    r = Routes(logits.device, T, n - identity, k, tile, shared)
    router = _lib.Router(n, k, identity, _ptr(bias), SCORES[scored], scale, int(as_scored))
    if on_input:
        assert not identity, "weights on the inputs go with experts that have rows"
        r.row_weights = torch.empty(r.tiles * tile, dtype=torch.float32, device=logits.device)
    check(lib().fb_route(ctypes.byref(router), logits.data_ptr(), T, logits.stride(0), tile, int(shared), r.weights.data_ptr(), r.ids.data_ptr(), r.slots.data_ptr(),
                         r.tile_expert.data_ptr(), r.live.data_ptr(), _ptr(r.row_weights), _stream()))
    count(1 if T <= 32 else 2)
    return r


def spread_rows(x, routes, out):
    """Each token's row of x into its choices' rows of out (fb_spread_rows)."""
    assert x.stride(1) == 1 and out.is_contiguous() and x.dtype == out.dtype
    size = x.element_size()
    check(lib().fb_spread_rows(x.data_ptr(), x.shape[0], x.shape[1] * size, x.stride(0) * size, routes.slots.data_ptr(), routes.k, out.data_ptr(), out.shape[0], _stream()))
    count()
    return out


def grouped(x, w, routes, out, kind=_lib.DENSE_NONE, shared=False, **extra):
    """Rows of tiles (shared: x's rows in every tile) by each tile's matrix of the batch w [n, K, N]: on the tensor cores
    where operands allow it (with a gated unit, if asked for; extra: its numbers); False where they do not."""
    n, K, N = w.shape
    if not (x.dtype == w.dtype == torch.bfloat16 and x.stride(1) == 1 and w.stride(1) == 1 and lib().fb_dense_supports(
            x.data_ptr(), x.stride(0), 0, w.data_ptr(), w.stride(2), w.stride(0) if n > 1 else 0, K, N, kind)):
        return False
    e = _lib.DenseEpilogue(kind=kind, **extra)
    check(lib().fb_dense_grouped(x.data_ptr(), x.shape[0], K, x.stride(0), int(shared), w.data_ptr(), N, w.stride(2), w.stride(0), n, routes.tile_expert.data_ptr(),
                                 routes.live.data_ptr(), routes.tiles, routes.tile, out.data_ptr(), _CODES[out.dtype], out.stride(0), ctypes.byref(e), _stream()))
    count()
    return True


def grouped_matmul(x, w, routes, out, shared=False, row_scale=None):
    """The same without a unit for any sizes, bf16 or fp32 (fb_grouped_matmul); row_scale: a number a row of the result."""
    n, K, N = w.shape
    assert x.stride(1) == 1 and out.stride(1) == 1
    check(lib().fb_grouped_matmul(_CODES[x.dtype], x.data_ptr(), x.shape[0], x.stride(0), int(shared), _CODES[w.dtype], w.data_ptr(), (ctypes.c_int64 * 3)(*w.stride()), n, K, N,
                                  routes.tile_expert.data_ptr(), routes.live.data_ptr(), routes.tiles, routes.tile, _ptr(row_scale), _CODES[out.dtype], out.data_ptr(), out.stride(0), _stream()))
    count()
    return out


def add_norm(x, x_out, mixer=None, mixer_scale=None, other=None, other_scale=None, chosen=None, routes=None, w=None, plus=0.0, eps=0.0, h=None,
             mixer_bias=None, own=None, gate=None, gate_bias=None, post=None):
    """A layer's end (fb_add_norm): x [T, cols] fp32 plus its branches (their sum gated and normed, where given) into x_out, and that normed by
    w + plus (w None: as it is) into h."""
    ld = lambda t: t.stride(0) if t is not None else 0
    of = lambda *ts: next((t.dtype for t in ts if t is not None), None)
    dtype = of(h, chosen) or torch.float32
    kind = of(mixer, other) or dtype if dtype == torch.bfloat16 else torch.float32
    assert all(t is None or t.dtype == kind for t in (mixer, other)) and all(t is None or t.dtype == dtype for t in (h, chosen, own))
    b = _lib.Branches(x.data_ptr(), ld(x), _ptr(mixer), ld(mixer), _ptr(mixer_scale), _ptr(other), ld(other), _ptr(other_scale), _ptr(chosen), ld(chosen),
                      _ptr(routes.slots) if routes else None, _ptr(routes.weights) if routes and getattr(routes, "row_weights", None) is None else None, routes.k if routes else 0, _ptr(x_out), ld(x_out), _ptr(w), plus, eps, _ptr(h), ld(h),
                      _ptr(mixer_bias), _ptr(own), ld(own), _ptr(gate), ld(gate), _ptr(gate_bias), _ptr(post))
    check(lib().fb_add_norm(ctypes.byref(b), x.shape[0], x.shape[1], _CODES[kind], _CODES[dtype], _stream()))
    count()

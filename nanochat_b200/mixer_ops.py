"""Entry points of libnckv for decoders that mix windowed attention with linear recurrences.

Same rules as ``ops``: shapes and dtypes are checked on the host, tensors must live on a CUDA device,
there is no CPU implementation.  Activations are bfloat16 or float32 (the exact mode); the residual
stream, norms, positions, scores and recurrent states are float32 in both.
"""
import contextlib

import torch

from . import _lib, ops

_scratch = {}  # (device index, stream) -> uint8 tensor for segmented recurrences


def _check(name, *tensors, dtypes=(torch.bfloat16, torch.float32)):
    ops._require_cuda(name, *tensors)
    for t in tensors:
        if t is not None and t.dtype not in dtypes:
            raise RuntimeError(f"nckv::{name}: unexpected dtype {t.dtype}")


def _ptr(t):
    return t.data_ptr() if t is not None else None


def _ctx(t):
    idx = t.device.index
    return idx, torch.cuda.current_stream(idx).cuda_stream


def _row_stride(name, t):
    """Row stride of (rows, C) activations that may be a column slice of a wider product."""
    if t.dim() != 2 or (t.size(1) > 1 and t.stride(1) != 1):
        raise RuntimeError(f"nckv::{name}: needs (rows, channels) with packed channels, got {tuple(t.shape)} / {t.stride()}")
    return t.stride(0) if t.size(0) > 1 else max(t.stride(0), t.size(1))


@contextlib.contextmanager
def full_precision_sums():
    """bf16 products keep fp32 partial sums, fp32 products stay fp32 (no TF32)."""
    m = torch.backends.cuda.matmul
    saved = m.allow_bf16_reduced_precision_reduction, m.allow_tf32
    m.allow_bf16_reduced_precision_reduction, m.allow_tf32 = False, False
    try:
        yield
    finally:
        m.allow_bf16_reduced_precision_reduction, m.allow_tf32 = saved


def product(a, w, f32_out=False):
    """a (rows, K) @ w (N, K)^T; bf16 operands can leave their fp32 sums unrounded."""
    if f32_out and a.dtype == torch.bfloat16:
        return torch.mm(a, w.t(), out_dtype=torch.float32)
    return torch.mm(a, w.t())


def add_product(y, a, w, y_scale=1.0, scale=1.0):
    """y_scale * y + scale * (a @ w^T) in fp32 (y fp32)."""
    if a.dtype == torch.bfloat16:
        return torch.addmm(y, a, w.t(), out_dtype=torch.float32, beta=y_scale, alpha=scale)
    return torch.addmm(y, a, w.t(), beta=y_scale, alpha=scale)


def resid_norm(x, y, weight, eps, dtype, B, T, tokens=None, table=None, want_h=False, final_weight=None, mu=None,
               carry=None):
    """One launch between two sublayers: ``x' = x + y / rms(y) * weight`` (``x`` None: ``table[tokens]``).
    Returns (x', h, mix): ``h`` is x' (or, with ``final_weight``, its norm) in ``dtype``; with ``mu``
    (n, W) and ``carry`` (B, W) ``mix`` is (n, rows, W), the token-shift mixes, and carry moves on.
    Without ``mu`` the stream is updated in place (and not stored at all before the last norm)."""
    name = "resid_norm"
    src = table if x is None else x
    W, rows = src.size(-1), B * T
    ops._require_cuda(name, x, y, weight, tokens, table, final_weight, mu, carry)
    dev = src.device
    for t, n in ((x, rows * W), (y, rows * W), (weight, W), (tokens, rows), (final_weight, W)):
        if t is not None and (t.numel() != n or not t.is_contiguous()):
            raise RuntimeError(f"nckv::{name}: operand of shape {tuple(t.shape)} does not fit {rows} rows of {W}")
    for t in (x, weight, final_weight, mu, carry):
        if t is not None and t.dtype != torch.float32:
            raise RuntimeError(f"nckv::{name}: the stream, norm weights and carried rows are float32, got {t.dtype}")
    if y is not None and y.dtype not in (dtype, torch.float32) or table is not None and table.dtype != dtype or \
            tokens is not None and tokens.dtype != torch.int64:
        raise RuntimeError(f"nckv::{name}: y / table must be {dtype} (y may be float32) and tokens int64")
    n_mix = 0
    if mu is not None:
        n_mix = mu.size(0)
        if mu.shape != (n_mix, W) or carry is None or carry.shape != (B, W) or not (mu.is_contiguous() and carry.is_contiguous()):
            raise RuntimeError(f"nckv::{name}: mu must be (n, {W}) and carry ({B}, {W})")
    h = torch.empty(rows, W, dtype=dtype, device=dev) if (want_h or final_weight is not None) else None
    mix = torch.empty(n_mix, rows, W, dtype=dtype, device=dev) if n_mix else None
    if final_weight is not None:
        x_out = None
    else:
        x_out = torch.empty(rows, W, dtype=torch.float32, device=dev) if (n_mix or x is None) else x
    idx, stream = _ctx(src)
    with ops._device_guard(idx):
        _lib.call("nckv_resid_norm", _ptr(x), _ptr(y), int(y is not None and y.dtype == torch.float32), _ptr(weight),
                  _ptr(tokens), _ptr(table), table.size(0) if table is not None else 0, _ptr(x_out), _ptr(h),
                  _ptr(final_weight), _ptr(mix), _ptr(mu), n_mix, _ptr(carry), B, T, W, float(eps),
                  int(dtype == torch.float32), stream)
    return x_out, h, mix


def silu_mul(gate_up):
    """silu(gate) * up over rows [gate | up]."""
    _check("silu_mul", gate_up)
    rows, two_f = gate_up.shape
    if not gate_up.is_contiguous() or two_f % 2:
        raise RuntimeError("nckv::silu_mul needs contiguous rows [gate | up]")
    out = torch.empty(rows, two_f // 2, dtype=gate_up.dtype, device=gate_up.device)
    idx, stream = _ctx(gate_up)
    with ops._device_guard(idx):
        _lib.call("nckv_silu_mul", _ptr(gate_up), _ptr(out), rows, two_f // 2, int(gate_up.dtype == torch.float32), stream)
    return out


def tanh_split(z, dtype):
    """tanh of fp32 rows (rows, R): float32 (rows, R), or bfloat16 (rows, 2 R) whose halves sum to it."""
    _check("tanh_split", z, dtypes=(torch.float32,))
    rows, R = z.shape
    f32 = dtype == torch.float32
    z = z.contiguous()
    out = torch.empty(rows, R if f32 else 2 * R, dtype=dtype, device=z.device)
    idx, stream = _ctx(z)
    with ops._device_guard(idx):
        _lib.call("nckv_tanh_split", _ptr(z), _ptr(out), rows, R, int(f32), stream)
    return out


def softcap(z, cap):
    """cap * tanh(z / cap) on fp32 logits, in place."""
    _check("softcap", z, dtypes=(torch.float32,))
    if not z.is_contiguous():
        raise RuntimeError("nckv::softcap needs a contiguous tensor")
    idx, stream = _ctx(z)
    with ops._device_guard(idx):
        _lib.call("nckv_softcap", _ptr(z), z.numel(), float(cap), stream)
    return z


def rope_unit_append(q, k, v, cos_sin, rot_dims, k_cache, v_cache, cache_seqlens, B, T, heads, kv_heads, dim, vdim,
                     q_scale, eps):
    """Rotate and unit-normalise q and k, append k and v to the cache; returns q' (B, T, heads, k_cache.size(3)).
    q, k, v: (B * T, heads * dim) rows, possibly column slices of one product."""
    name = "rope_unit_append"
    _check(name, q, k, v, k_cache, v_cache)
    ops._require_cuda(name, cos_sin, cache_seqlens)
    if not (q.dtype == k.dtype == v.dtype == k_cache.dtype == v_cache.dtype) or cache_seqlens.dtype != torch.int32 or \
            cos_sin.dtype != torch.float32 or not cos_sin.is_contiguous() or cos_sin.size(1) != rot_dims:
        raise RuntimeError(f"nckv::{name}: dtypes or table shape do not match")
    rows = B * T
    if q.shape != (rows, heads * dim) or k.shape != (rows, kv_heads * dim) or v.shape != (rows, kv_heads * vdim) or \
            k_cache.shape[:3] != v_cache.shape[:3] or k_cache.size(0) != B or k_cache.size(2) != kv_heads or \
            k_cache.size(3) < dim or v_cache.size(3) < vdim or cache_seqlens.numel() != B:
        raise RuntimeError(f"nckv::{name}: shapes do not match")
    for c in (k_cache, v_cache):
        if c.stride(3) != 1 or c.stride(2) != c.size(3):
            raise RuntimeError(f"nckv::{name}: cache heads must be packed")
    q_out = torch.empty(B, T, heads, k_cache.size(3), dtype=q.dtype, device=q.device)
    ws = ops.workspace(q.device, 1, 1, 1)
    idx, stream = _ctx(q)
    with ops._device_guard(idx):
        _lib.call("nckv_rope_unit_append", _ptr(q), _ptr(k), _ptr(v), _row_stride(name, q), _row_stride(name, k),
                  _row_stride(name, v), _ptr(cos_sin), _ptr(cache_seqlens), _ptr(q_out), _ptr(k_cache), _ptr(v_cache),
                  k_cache.stride(0), k_cache.stride(1), v_cache.stride(0), v_cache.stride(1), B, T, heads, kv_heads, dim,
                  vdim, k_cache.size(3), v_cache.size(3), rot_dims, cos_sin.size(0), k_cache.size(1), float(q_scale),
                  float(eps), int(q.dtype == torch.float32), _ptr(ws), stream)
    return q_out


def rms_rope_append(q, k, v, q_weight, k_weight, cos_sin, rot_dims, k_cache, v_cache, cache_seqlens, B, T, heads, kv_heads,
                    dim, vdim, q_scale, eps):
    """One weighted rms-norm over all of q's channels (and of k's), then rotation; k and v go to the cache.  k and v
    None: the cache holds another layer's keys, only q is made.  Returns q' (B, T, heads, k_cache.size(3))."""
    name = "rms_rope_append"
    _check(name, q, k, v, k_cache, v_cache)
    ops._require_cuda(name, q_weight, k_weight, cos_sin, cache_seqlens)
    if any(t is not None and t.dtype != q.dtype for t in (k, v, k_cache, v_cache)) or cache_seqlens.dtype != torch.int32 or \
            (rot_dims and (cos_sin.dtype != torch.float32 or not cos_sin.is_contiguous() or cos_sin.size(1) != rot_dims)):
        raise RuntimeError(f"nckv::{name}: dtypes or table shape do not match")
    rows = B * T
    if q.shape != (rows, heads * dim) or (k is None) != (v is None) or \
            (k is not None and (k.shape != (rows, kv_heads * dim) or v.shape != (rows, kv_heads * vdim))) or \
            k_cache.shape[:3] != v_cache.shape[:3] or k_cache.size(0) != B or k_cache.size(2) != kv_heads or \
            k_cache.size(3) < dim or v_cache.size(3) < vdim or cache_seqlens.numel() != B:
        raise RuntimeError(f"nckv::{name}: shapes do not match")
    for w, n in ((q_weight, heads * dim), (k_weight if k is not None else None, kv_heads * dim)):
        if w is not None and (w.dtype != torch.float32 or w.numel() != n or not w.is_contiguous()):
            raise RuntimeError(f"nckv::{name}: norm weights must be contiguous float32")
    for c in (k_cache, v_cache):
        if c.stride(3) != 1 or c.stride(2) != c.size(3):
            raise RuntimeError(f"nckv::{name}: cache heads must be packed")
    q_out = torch.empty(B, T, heads, k_cache.size(3), dtype=q.dtype, device=q.device)
    ws = ops.workspace(q.device, 1, 1, 1)
    idx, stream = _ctx(q)
    with ops._device_guard(idx):
        _lib.call("nckv_rms_rope_append", _ptr(q), _ptr(k), _ptr(v), _row_stride(name, q), _row_stride(name, k) if k is not None else 0,
                  _row_stride(name, v) if v is not None else 0, _ptr(q_weight), _ptr(k_weight), _ptr(cos_sin), _ptr(cache_seqlens),
                  _ptr(q_out), _ptr(k_cache), _ptr(v_cache), k_cache.stride(0), k_cache.stride(1), v_cache.stride(0),
                  v_cache.stride(1), B, T, heads, kv_heads, dim, vdim, k_cache.size(3), v_cache.size(3), rot_dims,
                  cos_sin.size(0) if rot_dims else 0, k_cache.size(1), float(q_scale), float(eps),
                  int(q.dtype == torch.float32), _ptr(ws), stream)
    return q_out


def _head_gate(name, gate, q):
    """(pointer, row stride) of a gate with one logit per token and head, or of none."""
    if gate is None:
        return None, 0
    if gate.dtype != q.dtype or gate.shape != (q.size(0) * q.size(1), q.size(2)):
        raise RuntimeError(f"nckv::{name}: the gate must be {q.dtype} ({q.size(0) * q.size(1)}, {q.size(2)}), got {tuple(gate.shape)}")
    return _ptr(gate), _row_stride(name, gate)


def window_attention(q, k_cache, v_cache, cache_seqlens, window, scale, sink=False, gate=None):
    """Attention over the ``window`` latest keys (None: all) for any head size, fp32 math; q: (B, T, heads, dim).
    ``sink``: one more term of score 0, without a value, in every softmax; ``gate`` (B * T, heads): every head's
    output times the sigmoid of its logit."""
    name = "window_attn"
    _check(name, q, k_cache, v_cache)
    B, T, H, dim = q.shape
    G, vdim = k_cache.size(2), v_cache.size(3)
    if not q.is_contiguous() or k_cache.size(3) != dim or k_cache.size(0) != B or H % G or q.dtype != k_cache.dtype or \
            v_cache.dtype != q.dtype or cache_seqlens.dtype != torch.int32:
        raise RuntimeError(f"nckv::{name}: q {tuple(q.shape)} does not fit the cache {tuple(k_cache.shape)}")
    out = torch.empty(B, T, H, vdim, dtype=q.dtype, device=q.device)
    gate_ptr, gate_stride = _head_gate(name, gate, q)
    idx, stream = _ctx(q)
    with ops._device_guard(idx):
        _lib.call("nckv_window_attn", _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(cache_seqlens), _ptr(out), k_cache.stride(0),
                  k_cache.stride(1), v_cache.stride(0), v_cache.stride(1), B, T, H, G, dim, vdim, k_cache.size(1),
                  1 << 30 if window is None else min(int(window), 1 << 30), float(scale), int(sink), gate_ptr, gate_stride,
                  int(q.dtype == torch.float32), stream)
    return out


def split_p_attention(q, k_cache, v_cache, cache_seqlens, window, sink=False, gate=None):
    """The 128-channel attention kernels with 16-bit probabilities (scores are scaled by 128 ** -0.5);
    q: (B, T, heads, 128) bf16 over a dense bf16 cache that already holds the new keys.  ``window``, ``sink`` and
    ``gate`` as in window_attention."""
    name = "attn_split_p"
    ops._require_cuda(name, q, k_cache, v_cache, cache_seqlens)
    ops._require_bf16(name, q, k_cache, v_cache)
    B, T, H, D = q.shape
    G = k_cache.size(2)
    if k_cache.shape != v_cache.shape or k_cache.stride() != v_cache.stride() or H % G or not q.is_contiguous() or \
            cache_seqlens.dtype != torch.int32:
        raise RuntimeError(f"nckv::{name}: q {tuple(q.shape)} does not fit the cache {tuple(k_cache.shape)}")
    sb, st = ops._cache_strides(name, k_cache)
    left = -1 if window is None else min(int(window) - 1, 1 << 30)
    gate_ptr, gate_stride = _head_gate(name, gate, q)
    out = torch.empty_like(q)
    idx, stream, ws = ops._launch_ctx(q, B, H, G)
    with ops._device_guard(idx):
        if T == 1:
            _lib.call("nckv_decode_attn_split_p", _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(cache_seqlens), _ptr(out), B, H, G,
                      D, k_cache.size(1), sb, st, 1, left, int(sink), gate_ptr, gate_stride, _ptr(ws), ws.numel(), stream)
        else:
            _lib.call("nckv_prefill_attn_split_p", _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(cache_seqlens), _ptr(out), B, T, H,
                      G, D, k_cache.size(1), sb, st, left, int(sink), gate_ptr, gate_stride, _ptr(ws), stream)
    return out


def recurrent(q, k, v, state, B, T, heads, dim, vdim, decay=None, decay_logits=None, decay_bias=None, bonus=None,
              gate=None, norm_weight=None, eps=0.0, silu_inputs=False):
    """Linear recurrence with a matrix state per head (see csrc/recurrent.cu); ``state`` (B, heads, dim, vdim)
    fp32 is updated in place.  Returns (B * T, heads * vdim): q's dtype when gated, else float32."""
    name = "recurrent"
    _check(name, q, k, v, gate)
    rows = B * T
    if q.shape != (rows, heads * dim) or k.shape != q.shape or v.shape != (rows, heads * vdim) or \
            state.shape != (B, heads, dim, vdim) or state.dtype != torch.float32 or not state.is_contiguous():
        raise RuntimeError(f"nckv::{name}: shapes do not match ({tuple(q.shape)}, {tuple(v.shape)}, state {tuple(state.shape)})")
    ops._require_cuda(name, state, decay, decay_logits, decay_bias, bonus, norm_weight)
    for t, n in ((decay, heads), (decay_bias, heads * dim), (bonus, heads * dim), (norm_weight, heads * vdim)):
        if t is not None and (t.dtype != torch.float32 or t.numel() != n or not t.is_contiguous()):
            raise RuntimeError(f"nckv::{name}: parameter vectors must be contiguous float32")
    if decay_logits is not None and (decay_logits.shape != (rows, heads * dim) or decay_logits.dtype != torch.float32):
        raise RuntimeError(f"nckv::{name}: decay_logits must be float32 ({rows}, {heads * dim})")
    if gate is not None and (gate.shape != v.shape or gate.dtype != q.dtype):
        raise RuntimeError(f"nckv::{name}: gate must look like v")
    out = torch.empty(rows, heads * vdim, dtype=q.dtype if norm_weight is not None else torch.float32, device=q.device)
    idx, stream = _ctx(q)
    with ops._device_guard(idx):
        need = _lib.lib.nckv_recurrent_workspace_bytes(B, T, heads, dim, vdim)
        ws = _scratch.get((idx, stream))
        if need and (ws is None or ws.numel() < need):
            ws = _scratch[(idx, stream)] = torch.empty(need, dtype=torch.uint8, device=q.device)
        _lib.call("nckv_recurrent", _ptr(q), _ptr(k), _ptr(v), _row_stride(name, q), _row_stride(name, k), _row_stride(name, v),
                  _ptr(decay_logits), _row_stride(name, decay_logits) if decay_logits is not None else 0, _ptr(decay_bias),
                  _ptr(bonus), _ptr(decay), _ptr(gate), _row_stride(name, gate) if gate is not None else 0,
                  _ptr(norm_weight), float(eps), _ptr(out), heads * vdim, _ptr(state), B, T, heads, dim, vdim,
                  int(silu_inputs), int(q.dtype == torch.float32), _ptr(ws), ws.numel() if ws is not None else 0, stream)
    return out


def gated_norm(x, gate, weight, group, eps, silu_gate=False):
    """x / rms(x) * weight * sigmoid(gate) (or silu(gate)), rms over groups of ``group`` channels; x fp32."""
    name = "gated_norm"
    _check(name, gate)
    rows, C = x.shape
    if x.dtype != torch.float32 or not x.is_contiguous() or gate.shape != x.shape or weight.dtype != torch.float32 or weight.numel() != C:
        raise RuntimeError(f"nckv::{name}: x and weight must be float32 and gate {tuple(x.shape)}")
    out = torch.empty(rows, C, dtype=gate.dtype, device=x.device)
    idx, stream = _ctx(x)
    with ops._device_guard(idx):
        _lib.call("nckv_gated_norm", _ptr(x), _ptr(gate), _row_stride(name, gate), _ptr(weight), _ptr(out), rows, C, group,
                  float(eps), int(silu_gate), int(gate.dtype == torch.float32), stream)
    return out


def _f32_vectors(name, *pairs):
    for t, n in pairs:
        if t is not None and (t.dtype != torch.float32 or t.numel() != n or not t.is_contiguous()):
            raise RuntimeError(f"nckv::{name}: parameters must be contiguous float32 of {n} elements, got {tuple(t.shape)} {t.dtype}")


def hyper_norm(x, y, hyper, into, weight, eps, dtype, tokens=None, table=None, streams=None, store=True):
    """One launch between two sublayers of a trunk with several residual streams x (rows, S, W) fp32.  ``hyper`` =
    (mix (S, S), out (S)) takes the last sublayer's output y ((rows, W), or (rows, parts, W) whose parts are
    added) into the streams; ``into`` (S, or None for ones) mixes them to the next input, which is
    layer-normed with ``weight``.  x None: all ``streams`` start as ``table[tokens]``.
    Returns (x', h); x is updated in place (``store`` False: not written)."""
    name = "hyper_norm"
    if x is None:
        S, W, n = streams, table.size(1), tokens.numel()
    else:
        n, S, W = x.shape
    ops._require_cuda(name, x, y, into, weight, tokens, table, *(hyper or ()))
    mix, out = hyper if y is not None else (None, None)
    _f32_vectors(name, (x, n * S * W), (mix, S * S), (out, S), (into, S), (weight, W))
    parts = 0
    if y is not None:
        parts = y.size(1) if y.dim() == 3 else 1
        if y.dtype != dtype or y.numel() != n * parts * W or not y.is_contiguous():
            raise RuntimeError(f"nckv::{name}: y {tuple(y.shape)} {y.dtype} does not fit {n} rows of {W}")
    if table is not None and (table.dtype != dtype or not table.is_contiguous() or tokens.dtype != torch.int64):
        raise RuntimeError(f"nckv::{name}: the table must be {dtype} and tokens int64")
    dev = weight.device
    h = torch.empty(n, W, dtype=dtype, device=dev)
    x_out = (torch.empty(n, S, W, dtype=torch.float32, device=dev) if x is None else x) if store else None
    idx, stream = _ctx(weight)
    with ops._device_guard(idx):
        _lib.call("nckv_hyper_norm", _ptr(x), _ptr(tokens), _ptr(table), table.size(0) if table is not None else 0, _ptr(y), parts,
                  _ptr(mix), _ptr(out), _ptr(into), _ptr(weight), _ptr(x_out), _ptr(h), n, S, W, float(eps),
                  int(dtype == torch.float32), stream)
    return x_out, h


def short_conv(x, taps, carry, B, T, in_bias=None, bias=None, silu=False):
    """Causal convolution per channel over rows x (B * T, C) (+ in_bias), taps (K, C) fp32 with the current token's last;
    ``carry`` (B, K - 1, C) fp32 holds the inputs before the call and is updated.  Returns (B * T, C)."""
    name = "short_conv"
    _check(name, x)
    rows, C = x.shape
    K = taps.size(0)
    ops._require_cuda(name, taps, carry, in_bias, bias)
    _f32_vectors(name, (taps, K * C), (carry, B * (K - 1) * C), (in_bias, C), (bias, C))
    if rows != B * T:
        raise RuntimeError(f"nckv::{name}: {rows} rows are not {B} x {T}")
    out = torch.empty(rows, C, dtype=x.dtype, device=x.device)
    idx, stream = _ctx(x)
    with ops._device_guard(idx):
        _lib.call("nckv_short_conv", _ptr(x), _row_stride(name, x), _ptr(taps), _ptr(in_bias), _ptr(bias), _ptr(carry), _ptr(out), B, T,
                  C, K, int(silu), int(x.dtype == torch.float32), stream)
    return out


def block_product(u, w, f32_out=True):
    """u (rows, blocks * n) times a square-block weight w (blocks, n, m): (blocks, rows, m)."""
    blocks, n, _ = w.shape
    parts = u.view(u.size(0), blocks, n).transpose(0, 1)
    if f32_out and u.dtype == torch.bfloat16:
        return torch.bmm(parts, w, out_dtype=torch.float32)
    return torch.bmm(parts, w)


def gated_scan(u, y, gates, gate_bias, y_bias, rate, state, B, T):
    """S = a S + sqrt(1 - a^2) sigmoid(i) u with a = exp(-rate sigmoid(r)); returns S * gelu_tanh(y + y_bias), (B * T, C).
    gates (blocks, B * T, 2 C / blocks) fp32: logits of r, then of i; gate_bias (2, C); state (B, C) is updated."""
    name = "gated_scan"
    _check(name, u, y)
    rows, C = u.shape
    blocks = gates.size(0)
    ops._require_cuda(name, gates, gate_bias, y_bias, rate, state)
    _f32_vectors(name, (gates, rows * 2 * C), (gate_bias, 2 * C), (y_bias, C), (rate, C), (state, B * C))
    if rows != B * T or y.shape != u.shape or y.dtype != u.dtype or gates.shape != (blocks, rows, 2 * (C // blocks)):
        raise RuntimeError(f"nckv::{name}: shapes do not match ({tuple(u.shape)}, {tuple(y.shape)}, gates {tuple(gates.shape)})")
    out = torch.empty(rows, C, dtype=u.dtype, device=u.device)
    need = _lib.lib.nckv_gated_scan_workspace_bytes(B, T, C)
    ws = torch.empty(need, dtype=torch.uint8, device=u.device) if need else None
    idx, stream = _ctx(u)
    with ops._device_guard(idx):
        _lib.call("nckv_gated_scan", _ptr(u), _row_stride(name, u), _ptr(y), _row_stride(name, y), _ptr(gates), _ptr(gate_bias),
                  _ptr(y_bias), _ptr(rate), _ptr(state), _ptr(out), B, T, C, blocks, int(u.dtype == torch.float32), _ptr(ws), need, stream)
    return out


def delta_rule(q, k, v, decay_logits, decay_bias, rate, beta_logits, state, B, T, heads, kv_heads, dim, vdim, gate, norm_weight, eps):
    """Gated delta rule (see csrc/delta.cu) with the heads' rms-norm, weight (vdim) and sigmoid gate behind it; ``state``
    (B, heads, dim, vdim) fp32 is updated.  Single tokens take one launch.  Returns (B * T, heads * vdim)."""
    name = "delta_rule"
    _check(name, q, k, v, beta_logits, gate)
    rows = B * T
    ops._require_cuda(name, decay_logits, decay_bias, rate, state, norm_weight)
    if q.shape != (rows, kv_heads * dim) or k.shape != q.shape or v.shape != (rows, heads * vdim) or gate.shape != v.shape or \
            beta_logits.shape != (rows, heads) or decay_logits.shape != (rows, heads * dim) or decay_logits.dtype != torch.float32 or \
            state.shape != (B, heads, dim, vdim) or any(t.dtype != q.dtype for t in (k, v, beta_logits, gate)):
        raise RuntimeError(f"nckv::{name}: shapes do not match ({tuple(q.shape)}, {tuple(v.shape)}, state {tuple(state.shape)})")
    _f32_vectors(name, (decay_bias, heads * dim), (rate, heads), (state, state.numel()), (norm_weight, vdim))
    f32 = int(q.dtype == torch.float32)
    inputs = (_ptr(q), _ptr(k), _ptr(v), _row_stride(name, q), _row_stride(name, k), _row_stride(name, v), _ptr(decay_logits),
              _row_stride(name, decay_logits), _ptr(decay_bias), _ptr(rate), _ptr(beta_logits), _row_stride(name, beta_logits))
    idx, stream = _ctx(q)
    quad = 4 * q.element_size()
    if T == 1 and vdim % 4 == 0 and vdim <= 128 and dim <= 1024 and not any(
            (t.data_ptr() | _row_stride(name, t) * t.element_size()) % quad for t in (v, gate)):
        out = torch.empty(rows, heads * vdim, dtype=q.dtype, device=q.device)
        with ops._device_guard(idx):
            _lib.call("nckv_delta_step", *inputs, _ptr(gate), _row_stride(name, gate), _ptr(norm_weight), float(eps), _ptr(out),
                      _ptr(state), B, heads, kv_heads, dim, vdim, f32, stream)
        return out
    out = torch.empty(rows, heads * vdim, dtype=torch.float32, device=q.device)
    chunks = not f32 and dim <= 128 and T > 4
    need = (_lib.lib.nckv_delta_chunk_workspace_bytes if chunks else _lib.lib.nckv_delta_workspace_bytes)(B, T, heads, dim)
    ws = torch.empty(need, dtype=torch.uint8, device=q.device)
    with ops._device_guard(idx):
        if chunks:
            status = ops.workspace(q.device, 1, 1, 1)
            _lib.call("nckv_delta_chunk", *inputs, _ptr(out), _ptr(state), B, T, heads, kv_heads, dim, vdim, _ptr(ws), need, _ptr(status), stream)
        else:
            _lib.call("nckv_delta_rule", *inputs, _ptr(out), _ptr(state), B, T, heads, kv_heads, dim, vdim, f32, _ptr(ws), need, stream)
    return gated_norm(out, gate, norm_weight.repeat(heads), vdim, eps)


class Routing:
    """(token, choice) pairs sorted by expert: pair ``slot[i]`` with weight ``scale[i]``, expert e at offsets[e] .. offsets[e + 1]."""

    def __init__(self, logits, top):
        name = "route"
        ops._require_cuda(name, logits)
        if logits.dim() != 2 or logits.dtype != torch.float32 or not logits.is_contiguous():
            raise RuntimeError(f"nckv::{name}: logits must be contiguous float32 (rows, experts)")
        rows, self.experts = logits.shape
        self.top, self.pairs, dev = top, rows * top, logits.device
        self.offsets = torch.empty(self.experts + 1, dtype=torch.int32, device=dev)
        self.slot = torch.empty(self.pairs, dtype=torch.int32, device=dev)
        self.scale = torch.empty(self.pairs, dtype=torch.float32, device=dev)
        need = _lib.lib.nckv_route_workspace_bytes(rows, self.experts, top)
        ws = torch.empty(need, dtype=torch.uint8, device=dev) if need else None
        idx, stream = _ctx(logits)
        with ops._device_guard(idx):
            _lib.call("nckv_route", _ptr(logits), _ptr(self.offsets), _ptr(self.slot), _ptr(self.scale), rows, self.experts, top,
                      _ptr(ws), need, stream)


def expert_product(a, w, routing, up):
    """up: a (rows, K) by w (experts, 2 N, K) to silu(s g) * (s u) in sorted order (pairs, N).  Else a (pairs, K) in sorted
    order by w (experts, N, K) to (rows, top, N)."""
    name = "experts"
    _check(name, a, w)
    E, n, K = w.shape
    rows = routing.pairs // routing.top
    N = n // 2 if up else n
    if a.shape != (rows if up else routing.pairs, K) or E != routing.experts or a.dtype != w.dtype or not (a.is_contiguous() and w.is_contiguous()):
        raise RuntimeError(f"nckv::{name}: a {tuple(a.shape)} does not fit w {tuple(w.shape)} and {routing.pairs} pairs")
    out = torch.empty((routing.pairs, N) if up else (rows, routing.top, N), dtype=a.dtype, device=a.device)
    ws = ops.workspace(a.device, 1, 1, 1)
    idx, stream = _ctx(a)
    with ops._device_guard(idx):
        _lib.call("nckv_experts", _ptr(a), _ptr(w), _ptr(out), _ptr(routing.offsets), _ptr(routing.slot), _ptr(routing.scale), int(up),
                  routing.pairs, E, routing.top, N, K, int(a.dtype == torch.float32), _ptr(ws), stream)
    return out

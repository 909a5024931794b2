"""Entry points of libnckv for decoders that mix windowed attention with linear recurrences.

Same rules as ``ops``: shapes and dtypes are checked on the host, tensors must live on a CUDA device,
there is no CPU implementation.  Activations are bfloat16 or float32 (the exact mode); the residual
stream, norms, positions, scores and recurrent states are float32 in both.
"""
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


def window_attention(q, k_cache, v_cache, cache_seqlens, window, scale):
    """Attention over the ``window`` latest keys for any head size, fp32 math; q: (B, T, heads, dim)."""
    name = "window_attn"
    _check(name, q, k_cache, v_cache)
    B, T, H, dim = q.shape
    G, vdim = k_cache.size(2), v_cache.size(3)
    if not q.is_contiguous() or k_cache.size(3) != dim or k_cache.size(0) != B or H % G or q.dtype != k_cache.dtype or \
            v_cache.dtype != q.dtype or cache_seqlens.dtype != torch.int32:
        raise RuntimeError(f"nckv::{name}: q {tuple(q.shape)} does not fit the cache {tuple(k_cache.shape)}")
    out = torch.empty(B, T, H, vdim, dtype=q.dtype, device=q.device)
    idx, stream = _ctx(q)
    with ops._device_guard(idx):
        _lib.call("nckv_window_attn", _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(cache_seqlens), _ptr(out), k_cache.stride(0),
                  k_cache.stride(1), v_cache.stride(0), v_cache.stride(1), B, T, H, G, dim, vdim, k_cache.size(1),
                  min(int(window), 1 << 30), float(scale), int(q.dtype == torch.float32), stream)
    return out


def split_p_attention(q, k_cache, v_cache, cache_seqlens, window):
    """The 128-channel attention kernels with 16-bit probabilities (scores are scaled by 128 ** -0.5);
    q: (B, T, heads, 128) bf16 over a dense bf16 cache that already holds the new keys."""
    name = "attn_split_p"
    ops._require_cuda(name, q, k_cache, v_cache, cache_seqlens)
    ops._require_bf16(name, q, k_cache, v_cache)
    B, T, H, D = q.shape
    G = k_cache.size(2)
    if k_cache.shape != v_cache.shape or k_cache.stride() != v_cache.stride() or H % G or not q.is_contiguous() or \
            cache_seqlens.dtype != torch.int32:
        raise RuntimeError(f"nckv::{name}: q {tuple(q.shape)} does not fit the cache {tuple(k_cache.shape)}")
    sb, st = ops._cache_strides(name, k_cache)
    left = min(int(window) - 1, 1 << 30)
    out = torch.empty_like(q)
    idx, stream, ws = ops._launch_ctx(q, B, H, G)
    with ops._device_guard(idx):
        if T == 1:
            _lib.call("nckv_decode_attn_split_p", _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(cache_seqlens), _ptr(out), B, H, G,
                      D, k_cache.size(1), sb, st, 1, left, _ptr(ws), ws.numel(), stream)
        else:
            _lib.call("nckv_prefill_attn_split_p", _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(cache_seqlens), _ptr(out), B, T, H,
                      G, D, k_cache.size(1), sb, st, left, _ptr(ws), stream)
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

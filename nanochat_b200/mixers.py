"""Sublayers that a decoder design can be put together from: sequence mixers and feed-forwards.

A mixer is built from its sizes and constants and a dict of weights, says what it keeps per sequence
(``declare``: key/value rows or fixed-size states in a ``HybridCache``), and maps activations of B rows
of T new tokens to the sublayer's output.  One forward serves prompts, portions of prompts and single
tokens; what the earlier tokens left is only read from the cache.  ``dtype`` is bfloat16, or float32 for
the exact mode; norms, positions, scores, decays and states are float32 in both.
"""
import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import mixer_ops as mo

TC_HEAD = 128    # head size of the tensor-core attention kernels; smaller heads are zero-padded to it
TC_GROUP = 16    # most query heads per key/value head they take
TC_ROWS = 1024   # most rows per decode launch


def rotary_table(length, dims, base, scaling=None, device=None):
    """(length, dims) fp32: cosines, then sines, of position * frequency for every pair, amplitude included.

    ``scaling`` (YaRN): pairs that turn often over the ``original`` context keep their frequency, slow ones
    are slowed by ``factor``, with a linear ramp over the pair index in between; the amplitude grows with
    the logarithm of the factor.  Computed in fp64 and rounded once."""
    half = dims // 2
    freq = base ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    amplitude = 1.0
    if scaling:
        factor, original = float(scaling["factor"]), float(scaling["original"])

        def pair_with(turns):
            return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

        lo = max(math.floor(pair_with(scaling["fast"])), 0)
        hi = min(math.ceil(pair_with(scaling["slow"])), dims - 1)
        slow = ((torch.arange(half, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        freq = freq / factor * slow + freq * (1 - slow)
        amplitude = 0.1 * math.log(factor) + 1.0
    angle = torch.outer(torch.arange(length, dtype=torch.float64, device=device), freq.to(device))
    return torch.cat([angle.cos() * amplitude, angle.sin() * amplitude], 1).float()


def f32(t):
    return t.float().contiguous()


@dataclass
class Rotary:
    dims: int
    base: float
    scaling: Optional[dict] = None

    def key(self):
        return (self.dims, self.base, tuple(sorted(self.scaling.items())) if self.scaling else None)


class WindowAttention:
    """Grouped-query attention over the latest ``window`` keys; q and k are rotated, then unit-normalised
    per head.  ``project`` weights are handed out by ``input_weights`` so that a layer can issue one
    product for several mixers that read the same activations."""

    def __init__(self, key, heads, kv_heads, dim, vdim, window, scale, rotary, weights, eps, dtype):
        assert heads % kv_heads == 0 and window > 0
        self.key, self.heads, self.kv_heads, self.dim, self.vdim = key, heads, kv_heads, dim, vdim
        self.window, self.scale, self.rotary, self.eps, self.dtype = window, scale, rotary, eps, dtype
        self.tensor_cores = (dtype == torch.bfloat16 and max(dim, vdim) <= TC_HEAD and heads // kv_heads <= TC_GROUP)
        self.k_width = TC_HEAD if self.tensor_cores else dim
        self.v_width = TC_HEAD if self.tensor_cores else vdim
        self.q_scale = scale * TC_HEAD ** 0.5 if self.tensor_cores else 1.0  # those kernels scale scores by 128 ** -0.5
        self._in = [weights["q"], weights["k"], weights["v"]]
        w_o = weights["o"]
        if self.v_width != vdim:  # the padded value channels meet zero columns
            w_o = torch.nn.functional.pad(w_o.view(-1, heads, vdim), (0, self.v_width - vdim)).reshape(w_o.size(0), -1)
        self.w_o = w_o.contiguous()

    def input_weights(self):
        return self._in

    def declare(self, cache):
        if self.tensor_cores and cache.batch_size > TC_ROWS:
            raise NotImplementedError(f"at most {TC_ROWS} rows per batch")
        cache.add_kv(self.key, self.kv_heads, self.k_width, self.v_width, self.dtype)
        cache.add_table(self.rotary.key(), lambda n, dev: rotary_table(n, self.rotary.dims, self.rotary.base,
                                                                     self.rotary.scaling, dev))

    def attend(self, q, k, v, cache, B, T):
        """Head outputs (B * T, heads * v_width) before the output projection."""
        kc, vc = cache.kv[self.key]
        q = mo.rope_unit_append(q, k, v, cache.tables[self.rotary.key()], self.rotary.dims, kc, vc, cache.cache_seqlens, B, T,
                                self.heads, self.kv_heads, self.dim, self.vdim, self.q_scale, self.eps)
        if self.tensor_cores:
            y = mo.split_p_attention(q, kc, vc, cache.cache_seqlens, self.window)
        else:
            y = mo.window_attention(q, kc, vc, cache.cache_seqlens, self.window, self.scale)
        return y.view(B * T, -1)


class ScaledLinearAttention:
    """Linear attention with one decay constant per head (silu on q, k and v), an rms-norm over all heads
    together and a sigmoid gate."""

    def __init__(self, key, heads, dim, vdim, decay, weights, eps, dtype):
        assert len(decay) == heads
        self.key, self.heads, self.dim, self.vdim, self.eps, self.dtype = key, heads, dim, vdim, eps, dtype
        self._in = [weights["q"], weights["k"], weights["v"], weights["g"]]
        self.w_o, self.norm = weights["o"], f32(weights["norm"])
        self.decay = torch.tensor(decay, dtype=torch.float32, device=self.norm.device)

    def input_weights(self):
        return self._in

    def declare(self, cache):
        cache.add_state(self.key, (self.heads, self.dim, self.vdim))

    def attend(self, q, k, v, gate, cache, B, T):
        o = mo.recurrent(q, k, v, cache.state[self.key], B, T, self.heads, self.dim, self.vdim, decay=self.decay,
                         silu_inputs=True)
        return mo.gated_norm(o, gate, self.norm, self.heads * self.vdim, self.eps)


class ParallelMixer:
    """Two mixers on the same activations, their outputs added with a factor each: windowed attention on
    the left, scaled linear attention on the right.  One product makes all their inputs."""

    shift = None  # reads the activations themselves

    def __init__(self, left, right, left_scale, right_scale):
        self.left, self.right, self.left_scale, self.right_scale = left, right, left_scale, right_scale
        ws = left.input_weights() + right.input_weights()
        self.widths = [w.size(0) for w in ws]
        self.w_in = torch.cat(ws, 0).contiguous()
        left._in = right._in = None

    def declare(self, cache):
        self.left.declare(cache)
        self.right.declare(cache)

    def __call__(self, h, cache, B, T):
        lq, lk, lv, rq, rk, rv, rg = mo.product(h, self.w_in).split(self.widths, 1)
        y = mo.product(self.left.attend(lq, lk, lv, cache, B, T), self.left.w_o, f32_out=True)
        return mo.add_product(y, self.right.attend(rq, rk, rv, rg, cache, B, T), self.right.w_o, self.left_scale,
                              self.right_scale)


class WkvMixer:
    """RWKV-style time mixing: five token-shift mixes, a decay per token and key channel from a low-rank
    path, a bonus for the current token, a norm per head and a silu gate."""

    MIXES = "rkvgw"

    def __init__(self, key, heads, dim, weights, eps, dtype):
        self.key, self.heads, self.dim, self.eps, self.dtype = key, heads, dim, eps, dtype
        self.shift = f32(torch.stack([weights["mu." + s] for s in self.MIXES]))
        self.w_rkvg = torch.stack([weights[s] for s in "rkvg"]).contiguous()
        self.w1 = weights["w1"]
        # the tanh between the two low-rank products enters the second one as two bf16 terms
        self.w2 = weights["w2"] if dtype == torch.float32 else torch.cat([weights["w2"]] * 2, 1).contiguous()
        self.w0, self.bonus, self.norm = f32(weights["w0"]), f32(weights["u"]), f32(weights["norm"])
        self.w_o = weights["o"]
        self.width = self.w1.size(1)
        self.gate_in_kernel = dim <= 128

    def declare(self, cache):
        cache.add_state(self.key, (self.heads, self.dim, self.dim))
        cache.add_state(self.key + ".shift", (self.width,))

    def carry(self, cache):
        return cache.state[self.key + ".shift"]

    def __call__(self, mix, cache, B, T):
        r, k, v, g = torch.bmm(mix[:4], self.w_rkvg.transpose(1, 2)).unbind(0)
        low = mo.tanh_split(mo.product(mix[4], self.w1, f32_out=True), self.dtype)
        args = dict(decay_logits=mo.product(low, self.w2, f32_out=True), decay_bias=self.w0, bonus=self.bonus)
        state = cache.state[self.key]
        if self.gate_in_kernel:
            o = mo.recurrent(r, k, v, state, B, T, self.heads, self.dim, self.dim, gate=g, norm_weight=self.norm,
                             eps=self.eps, **args)
        else:
            o = mo.recurrent(r, k, v, state, B, T, self.heads, self.dim, self.dim, **args)
            o = mo.gated_norm(o, g, self.norm, self.dim, self.eps, silu_gate=True)
        return mo.product(o, self.w_o)


class GatedFeedForward:
    """W_down (silu(W_gate h) * (W_up h)), gate and up in one product."""

    def __init__(self, weights):
        self.w_in = torch.cat([weights["gate"], weights["up"]], 0).contiguous()
        self.w_down = weights["down"]

    def __call__(self, h):
        return mo.product(mo.silu_mul(mo.product(h, self.w_in)), self.w_down)

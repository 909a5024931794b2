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


def yarn_scaling(freq, dims, base, scaling):
    """(frequencies, amplitude): pairs that turn often over the ``original`` context keep their frequency, slow ones
    are slowed by ``factor``, with a linear ramp over the pair index in between; the amplitude grows with the
    logarithm of the factor."""
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_with(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(pair_with(scaling["fast"])), 0)
    hi = min(math.ceil(pair_with(scaling["slow"])), dims - 1)
    slow = ((torch.arange(freq.numel(), dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return freq / factor * slow + freq * (1 - slow), 0.1 * math.log(factor) + 1.0


def banded_scaling(freq, scaling):
    """Frequencies in three bands by how often a pair turns over the ``original`` context: ``high`` times or more
    often keeps it, ``low`` times or less is slowed by ``factor``, in between the two are mixed by the turns."""
    turns = float(scaling["original"]) * freq / (2 * math.pi)
    low, high = float(scaling["low"]), float(scaling["high"])
    keep = ((turns - low) / (high - low)).clamp(0, 1) if high > low else (turns >= low).double()
    return (1 - keep) * freq / float(scaling["factor"]) + keep * freq


def rotary_table(length, dims, base, scaling=None, device=None):
    """(length, dims) fp32: cosines, then sines, of position * frequency for every pair, amplitude included.
    ``scaling``: YaRN's constants (factor, original, fast, slow), or the three bands' (factor, original, low,
    high).  Computed in fp64 and rounded once."""
    freq = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    amplitude = 1.0
    if scaling and "low" in scaling:
        freq = banded_scaling(freq, scaling)
    elif scaling:
        freq, amplitude = yarn_scaling(freq, dims, base, scaling)
    angle = torch.outer(torch.arange(length, dtype=torch.float64, device=device), freq.to(device))
    return torch.cat([angle.cos() * amplitude, angle.sin() * amplitude], 1).float()


def f32(t):
    return t.float().contiguous()


def stacked(weights, multiple=8):
    """One weight for several products of the same input, (weight, widths); zero rows fill it up to a multiple of
    ``multiple`` outputs, so that the rows of the result stay aligned."""
    widths = [w.size(0) for w in weights]
    rest = -sum(widths) % multiple
    if rest:
        weights = list(weights) + [weights[0].new_zeros(rest, weights[0].size(1))]
    return torch.cat(weights, 0).contiguous(), widths


def columns(t, widths):
    """Consecutive column slices of a product."""
    out, at = [], 0
    for n in widths:
        out.append(t[:, at:at + n])
        at += n
    return out


@dataclass
class Rotary:
    dims: int
    base: float
    scaling: Optional[dict] = None

    def key(self):
        return (self.dims, self.base, tuple(sorted(self.scaling.items())) if self.scaling else None)


class CachedAttention:
    """What the attention mixers share: heads on the tensor-core kernels where sizes allow (zero-padded to their
    width), key/value rows and the rotary table in the cache.  ``window`` None: all earlier keys."""

    def __init__(self, key, heads, kv_heads, dim, vdim, window, scale, rotary, w_o, eps, dtype):
        assert heads % kv_heads == 0 and (window is None or window > 0)
        self.key, self.heads, self.kv_heads, self.dim, self.vdim = key, heads, kv_heads, dim, vdim
        self.window, self.scale, self.rotary, self.eps, self.dtype = window, scale, rotary, eps, dtype
        self.tensor_cores = (dtype == torch.bfloat16 and max(dim, vdim) <= TC_HEAD and heads // kv_heads <= TC_GROUP)
        self.k_width = TC_HEAD if self.tensor_cores else dim
        self.v_width = TC_HEAD if self.tensor_cores else vdim
        self.q_scale = scale * TC_HEAD ** 0.5 if self.tensor_cores else 1.0  # those kernels scale scores by 128 ** -0.5
        if self.v_width != vdim:  # the padded value channels meet zero columns
            w_o = torch.nn.functional.pad(w_o.view(-1, heads, vdim), (0, self.v_width - vdim)).reshape(w_o.size(0), -1)
        self.w_o = w_o.contiguous()

    def declare(self, cache, own_kv=True):
        if self.tensor_cores and cache.batch_size > TC_ROWS:
            raise NotImplementedError(f"at most {TC_ROWS} rows per batch")
        if own_kv:
            cache.add_kv(self.key, self.kv_heads, self.k_width, self.v_width, self.dtype)
        cache.add_table(self.rotary.key(), lambda n, dev: rotary_table(n, self.rotary.dims, self.rotary.base,
                                                                     self.rotary.scaling, dev))

    def over_cache(self, q, kc, vc, cache, B, T, **end):
        """Head outputs (B * T, heads * v_width) of rotated queries over rows that hold the new keys already."""
        if self.tensor_cores:
            y = mo.split_p_attention(q, kc, vc, cache.cache_seqlens, self.window, **end)
        else:
            y = mo.window_attention(q, kc, vc, cache.cache_seqlens, self.window, self.scale, **end)
        return y.view(B * T, -1)


class WindowAttention(CachedAttention):
    """Grouped-query attention over the latest ``window`` keys; q and k are rotated, then unit-normalised
    per head.  ``project`` weights are handed out by ``input_weights`` so that a layer can issue one
    product for several mixers that read the same activations."""

    def __init__(self, key, heads, kv_heads, dim, vdim, window, scale, rotary, weights, eps, dtype):
        super().__init__(key, heads, kv_heads, dim, vdim, window, scale, rotary, weights["o"], eps, dtype)
        self._in = [weights["q"], weights["k"], weights["v"]]

    def input_weights(self):
        return self._in

    def attend(self, q, k, v, cache, B, T):
        """Head outputs (B * T, heads * v_width) before the output projection."""
        kc, vc = cache.kv[self.key]
        q = mo.rope_unit_append(q, k, v, cache.tables[self.rotary.key()], self.rotary.dims, kc, vc, cache.cache_seqlens, B, T,
                                self.heads, self.kv_heads, self.dim, self.vdim, self.q_scale, self.eps)
        return self.over_cache(q, kc, vc, cache, B, T)


class GatedAttention(CachedAttention):
    """Grouped-query attention with a weighted rms-norm over the whole of q and of k ahead of the rotation, an
    optional sink in the softmax and a sigmoid gate per head.  ``source``: another GatedAttention whose keys and
    values are used instead of own ones (its layer runs earlier in the same forward)."""

    shift = None  # reads the activations themselves

    def __init__(self, key, heads, kv_heads, dim, vdim, window, scale, rotary, sink, weights, eps, dtype, source=None):
        super().__init__(key, heads, kv_heads, dim, vdim, window, scale, rotary, weights["o"], eps, dtype)
        self.sink, self.source = sink, source
        if source is not None and (source.kv_heads, source.k_width, source.v_width) != (kv_heads, self.k_width, self.v_width):
            raise ValueError(f"{key}: the keys and values of {source.key} have other sizes")
        self.norm_q = f32(weights["q.norm"])
        self.norm_k = f32(weights["k.norm"]) if source is None else None
        names = "qkvg" if source is None else "qg"
        self.w_in, self.widths = stacked([weights[s] for s in names])

    def declare(self, cache):
        super().declare(cache, own_kv=self.source is None)

    def __call__(self, h, cache, B, T):
        parts = columns(mo.product(h, self.w_in), self.widths)
        q, gate = parts[0], parts[-1]
        k, v = parts[1:3] if self.source is None else (None, None)
        kc, vc = cache.kv[(self.source or self).key]
        q = mo.rms_rope_append(q, k, v, self.norm_q, self.norm_k, cache.tables[self.rotary.key()], self.rotary.dims, kc, vc,
                               cache.cache_seqlens, B, T, self.heads, self.kv_heads, self.dim, self.vdim, self.q_scale, self.eps)
        return mo.product(self.over_cache(q, kc, vc, cache, B, T, sink=self.sink, gate=gate), self.w_o)


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


class ShortConv:
    """Causal convolution per channel over the projections of a mixer; the last inputs are part of its state."""

    def __init__(self, key, taps, in_bias=None, bias=None, silu=False):
        self.key, self.silu = key, silu
        self.taps = f32(taps.t())  # tap-major
        self.in_bias = f32(in_bias) if in_bias is not None else None
        self.bias = f32(bias) if bias is not None else None

    def declare(self, cache):
        cache.add_state(self.key, (self.taps.size(0) - 1, self.taps.size(1)))

    def __call__(self, x, cache, B, T):
        return mo.short_conv(x, self.taps, cache.state[self.key], B, T, self.in_bias, self.bias, self.silu)


class RealGatedRecurrence:
    """Two branches: a gelu gate, and a short convolution into a linear recurrence over channels whose decay and
    input gate come from block-diagonal products (``sharpness`` scales the logarithm of the decay)."""

    shift = None

    def __init__(self, key, width, blocks, conv, weights, dtype, sharpness=8.0):
        self.key, self.width = key, width
        if weights["conv"].size(1) != conv:
            raise ValueError(f"{key}: the filters have {weights['conv'].size(1)} taps, the configuration says {conv}")
        self.w_in, self.widths = stacked([weights["y"], weights["x"]])
        self.conv = ShortConv(key + ".conv", weights["conv"], weights["x.b"], weights["conv.b"])
        # (blocks, n, 2 n): logits of the decay gate, then of the input gate
        self.w_gates = torch.cat([weights["ra"].transpose(1, 2), weights["ri"].transpose(1, 2)], 2).contiguous()
        self.gate_bias = torch.stack([f32(weights["ra.b"]).view(-1), f32(weights["ri.b"]).view(-1)])
        self.y_bias = f32(weights["y.b"])
        self.rate = (sharpness * torch.nn.functional.softplus(weights["lam"].double())).float()
        self.w_o = weights["o"]

    def declare(self, cache):
        cache.add_state(self.key, (self.width,))
        self.conv.declare(cache)

    def __call__(self, h, cache, B, T):
        y, x = columns(mo.product(h, self.w_in), self.widths)
        u = self.conv(x, cache, B, T)
        o = mo.gated_scan(u, y, mo.block_product(u, self.w_gates), self.gate_bias, self.y_bias, self.rate, cache.state[self.key], B, T)
        return mo.product(o, self.w_o)


class DeltaMixer:
    """Gated delta rule with a decay per head and key channel from a low-rank path; q, k and v pass a short
    convolution and silu; each head's output is normed and gated by a second low-rank path."""

    shift = None

    def __init__(self, key, heads, kv_heads, dim, vdim, conv, weights, eps, dtype):
        assert heads % kv_heads == 0
        self.key, self.heads, self.kv_heads, self.dim, self.vdim, self.eps = key, heads, kv_heads, dim, vdim, eps
        if any(weights[s + ".conv"].size(1) != conv for s in "qkv"):
            raise ValueError(f"{key}: the configuration says {conv} taps")
        self.w_in, widths = stacked([weights[s] for s in ("q", "k", "v", "a1", "g1", "b")])
        self.qkv = widths[:3]
        self.widths = [sum(self.qkv)] + widths[3:]
        self.conv = ShortConv(key + ".conv", torch.cat([weights[s + ".conv"] for s in "qkv"]), silu=True)
        self.w_decay, self.w_gate = weights["a2"], weights["g2"]
        self.rate = torch.exp(weights["A_log"].double()).float()
        self.dt_bias, self.norm, self.w_o = f32(weights["dt_bias"]), f32(weights["norm"]), weights["o"]

    def declare(self, cache):
        cache.add_state(self.key, (self.heads, self.dim, self.vdim))
        self.conv.declare(cache)

    def __call__(self, h, cache, B, T):
        qkv, a, g, beta = columns(mo.product(h, self.w_in), self.widths)
        q, k, v = columns(self.conv(qkv, cache, B, T), self.qkv)
        o = mo.delta_rule(q, k, v, mo.product(a, self.w_decay, f32_out=True), self.dt_bias, self.rate, beta, cache.state[self.key],
                          B, T, self.heads, self.kv_heads, self.dim, self.vdim, mo.product(g, self.w_gate), self.norm, self.eps)
        return mo.product(o, self.w_o)


class ExpertsFeedForward:
    """Mixture of gated feed-forwards: a token goes to the ``top`` experts with the largest sigmoid scores, and the
    score multiplies the expert's input.  Returns (rows, top, width), still to be added up."""

    def __init__(self, weights, experts, top):
        assert 0 < top <= experts
        self.top = top
        self.router = weights["router"]
        self.w_in = torch.stack([torch.cat([weights[f"e{e}.gate"], weights[f"e{e}.up"]]) for e in range(experts)]).contiguous()
        self.w_down = torch.stack([weights[f"e{e}.down"] for e in range(experts)]).contiguous()

    def __call__(self, h):
        routing = mo.Routing(mo.product(h, self.router, f32_out=True), self.top)
        return mo.expert_product(mo.expert_product(h, self.w_in, routing, up=True), self.w_down, routing, up=False)

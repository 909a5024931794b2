"""Zuvulorn: a decoder of several residual streams whose layers are put together from a list in its configuration.

Mixers: ``rglru`` (real-gated linear recurrence), ``attention`` (grouped-query attention with a sink and head
gates, on its own keys and values or on an earlier layer's) and ``channel_delta`` (gated delta rule).  A layer
may have a feed-forward, a mixture of experts.  Around every sublayer the streams are mixed (hyper-
connections); its input is layer-normed.  Sizes come from the configuration or the tensors' shapes.
"""
from dataclasses import dataclass, field
from typing import List

import torch

from . import mixer_ops as mo
from .hybrid import HybridDecoder, Scope
from .mixers import DeltaMixer, ExpertsFeedForward, GatedAttention, RealGatedRecurrence, Rotary, f32
from .models import register


@dataclass
class ZuvulornConfig:
    vocab_size: int
    n_embd: int
    eps: float
    streams: int
    layers: List[dict] = field(repr=False)
    sequence_len: int = 4096  # default capacity of a generation without max_tokens; the design itself has no limit

    @property
    def n_layer(self):
        return len(self.layers)

    @classmethod
    def from_dict(cls, c):
        for i, layer in enumerate(c["layers"]):
            if layer["type"] not in ("rglru", "attention", "channel_delta"):
                raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            j = layer["mixer"].get("kv_from")
            if j is not None and not (0 <= j < i and c["layers"][j]["type"] == "attention"
                                      and c["layers"][j]["mixer"].get("kv_from") is None):
                raise ValueError(f"layer {i}: layer {j} has no keys and values to share")
        return cls(c["vocab"], c["width"], c["norm"]["eps"], c["streams"], c["layers"])


def tensor_shapes(config, rank):
    """name -> shape of every tensor of a configuration (a dict as in config.json); ``rank`` is the inner width
    of the low-rank paths, which the configuration leaves to the tensors."""
    W, S = config["width"], config["streams"]
    shapes = {"embed": (config["vocab"], W), "final.norm": (W,), "head": (config["vocab"], W)}
    for i, layer in enumerate(config["layers"]):
        m, p, sublayers = layer["mixer"], f"l{i}.", [1]
        mix = {}
        if layer["type"] == "rglru":
            n, part = m["width"], (m["blocks"], m["width"] // m["blocks"])
            mix = {"y": (n, W), "y.b": (n,), "x": (n, W), "x.b": (n,), "conv": (n, m["conv"]), "conv.b": (n,), "lam": (n,),
                   "ra": part + part[1:], "ra.b": part, "ri": part + part[1:], "ri.b": part, "o": (W, n)}
        elif layer["type"] == "attention":
            nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            mix = {"q": (nq, W), "q.norm": (nq,), "g": (m["heads"], W), "o": (W, m["heads"] * m["vdim"])}
            if m.get("kv_from") is None:
                mix.update({"k": (nk, W), "k.norm": (nk,), "v": (m["kv_heads"] * m["vdim"], W)})
        else:
            nk, nd, nv = m["kv_heads"] * m["dim"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            mix = {"q": (nk, W), "k": (nk, W), "v": (nv, W), "q.conv": (nk, m["conv"]), "k.conv": (nk, m["conv"]),
                   "v.conv": (nv, m["conv"]), "b": (m["heads"], W), "A_log": (m["heads"],), "dt_bias": (nd,), "norm": (m["vdim"],),
                   "a1": (rank, W), "a2": (nd, rank), "g1": (rank, W), "g2": (nv, rank), "o": (W, nv)}
        shapes.update({f"{p}mix.{k}": v for k, v in mix.items()})
        if layer.get("mlp") is not None:
            sublayers.append(2)
            ff, n = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]["experts"]
            shapes[p + "mlp.router"] = (n, W)
            for e in range(n):
                shapes.update({f"{p}mlp.e{e}.gate": (ff, W), f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
        for q in sublayers:
            shapes.update({f"{p}norm{q}": (W,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
    return shapes


class _Sublayer:
    """The norm of a sublayer's input and how it sits between the streams."""

    def __init__(self, tensors, p, q):
        self.norm = f32(tensors[f"{p}norm{q}"])
        self.into = f32(tensors[f"{p}hc{q}.in"])
        self.back = f32(tensors[f"{p}hc{q}.mix"]), f32(tensors[f"{p}hc{q}.out"])


class _Layer:
    def __init__(self, i, spec, tensors, eps, dtype, earlier):
        p, m, kind = f"l{i}.", spec["mixer"], spec["type"]
        mix = Scope(tensors, p + "mix.")
        if kind == "rglru":
            self.mixer = RealGatedRecurrence(p + kind, m["width"], m["blocks"], m["conv"], mix, dtype)
        elif kind == "attention":
            rot, j = m.get("rot"), m.get("kv_from")
            rotary = Rotary(rot["dims"], rot["base"], rot.get("scaling")) if rot else Rotary(0, 1.0)
            self.mixer = GatedAttention(p + kind, m["heads"], m["kv_heads"], m["dim"], m["vdim"], None, m["scale"], rotary, True, mix, eps,
                                        dtype, source=earlier[j].mixer if j is not None else None)
        else:
            self.mixer = DeltaMixer(p + kind, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], mix, eps, dtype)
        self.around_mixer, self.ff = _Sublayer(tensors, p, 1), None
        if spec.get("mlp") is not None:
            router = spec["mlp"]["router"]
            self.ff = ExpertsFeedForward(Scope(tensors, p + "mlp."), router["experts"], router["top"])
            self.around_ff = _Sublayer(tensors, p, 2)


@register("Zuvulorn")
class Zuvulorn(HybridDecoder):
    def __init__(self, config, tensors, dtype=torch.bfloat16):
        self.config, self.dtype = config, dtype
        self.embed, self.head = tensors["embed"], tensors["head"]
        self.layers = []
        for i, spec in enumerate(config.layers):
            self.layers.append(_Layer(i, spec, tensors, config.eps, dtype, self.layers))
        self.final_norm = f32(tensors["final.norm"])

    parse = staticmethod(ZuvulornConfig.from_dict)
    shapes = staticmethod(lambda config: tensor_shapes(config, rank=None))

    @torch.inference_mode()
    def forward(self, idx, targets=None, kv_cache=None, logits_at=None, on_layer=None):
        """fp32 logits (B, T, vocab), or (B, len(logits_at), vocab) at the given places of the T tokens (an empty
        list runs the tokens and returns None).  ``on_layer(i, x)`` sees the sum of the streams after each layer."""
        B, T, kv_cache = self.begin(idx, targets, kv_cache)
        common = dict(eps=self.config.eps, dtype=self.dtype)
        with mo.full_precision_sums():
            x = y = back = None
            source = dict(tokens=idx.contiguous().view(-1), table=self.embed, streams=self.config.streams)
            for i, layer in enumerate(self.layers):
                at = layer.around_mixer
                x, h = mo.hyper_norm(x, y, back, at.into, at.norm, **source, **common)
                source = {}
                if on_layer is not None and i > 0:
                    on_layer(i - 1, x.sum(1))
                y, back = layer.mixer(h, kv_cache, B, T), at.back
                if layer.ff is not None:
                    at = layer.around_ff
                    x, h = mo.hyper_norm(x, y, back, at.into, at.norm, **common)
                    y, back = layer.ff(h), at.back
            if on_layer is not None:
                on_layer(self.config.n_layer - 1, mo.hyper_norm(x.clone(), y, back, None, self.final_norm, **common)[0].sum(1))
            kv_cache.advance(T)
            n = T
            if logits_at is not None:
                if len(logits_at) == 0:
                    return None
                n = len(logits_at)
                x, y = self.pick(x, B, T, logits_at), self.pick(y, B, T, logits_at)
            _, h = mo.hyper_norm(x, y, back, None, self.final_norm, store=False, **common)
            logits = mo.product(h, self.head, f32_out=True)
        return logits.view(B, n, -1)

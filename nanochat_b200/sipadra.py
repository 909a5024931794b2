"""Sipadra: a decoder whose layers are put together from a list in its configuration.

Residual stream in 32-bit; a layer adds the rms-normed output of its mixer (``wkv``: RWKV-style time
mixing, ``parallel``: windowed attention beside scaled linear attention) and then that of its gated
feed-forward, if it has one.  Sublayers read the stream itself.  The output head is the embedding
table, with a soft cap on the logits.  Sizes come from the configuration or the tensors' shapes.
"""
from dataclasses import dataclass, field
from typing import List, Optional

import torch

from . import mixer_ops as mo
from .hybrid import HybridDecoder, Scope
from .mixers import GatedFeedForward, ParallelMixer, Rotary, ScaledLinearAttention, WindowAttention, WkvMixer, f32
from .models import register


@dataclass
class SipadraConfig:
    vocab_size: int
    n_embd: int
    eps: float
    logit_softcap: Optional[float]
    layers: List[dict] = field(repr=False)
    sequence_len: int = 4096  # default capacity of a generation without max_tokens; the design itself has no limit

    @property
    def n_layer(self):
        return len(self.layers)

    @classmethod
    def from_dict(cls, c):
        for i, layer in enumerate(c["layers"]):
            if layer["type"] not in ("wkv", "parallel"):
                raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        return cls(c["vocab"], c["width"], c["norm"]["eps"], c.get("logit_softcap"), c["layers"])


def tensor_shapes(config, rank):
    """name -> shape of every tensor of a configuration (a dict as in config.json); ``rank`` is the inner width
    of the decay paths, which the configuration leaves to the tensors."""
    W = config["width"]
    shapes = {"embed": (config["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        shapes[p + "norm1"] = (W,)
        if layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            shapes.update({f"{p}mix.mu.{s}": (W,) for s in WkvMixer.MIXES})
            shapes.update({f"{p}mix.{s}": (n, W) for s in "rkvg"})
            shapes.update({p + "mix.w1": (rank, W), p + "mix.w2": (n, rank), p + "mix.w0": (n,),
                           p + "mix.u": (m["heads"], m["dim"]), p + "mix.norm": (n,), p + "mix.o": (W, n)})
        else:
            a, b, left, right = m["left"], m["right"], p + "mix.left.", p + "mix.right."
            out, n = a["heads"] * a["vdim"], b["heads"] * b["vdim"]
            shapes.update({left + "q": (a["heads"] * a["dim"], W), left + "k": (a["kv_heads"] * a["dim"], W),
                           left + "v": (a["kv_heads"] * a["vdim"], W), left + "o": (W, out),
                           right + "q": (b["heads"] * b["dim"], W), right + "k": (b["heads"] * b["dim"], W),
                           right + "v": (n, W), right + "g": (n, W), right + "norm": (n,), right + "o": (W, n)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            shapes.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return shapes


class _Layer:
    def __init__(self, i, spec, tensors, eps, dtype):
        p, m = f"l{i}.", spec["mixer"]
        mix = Scope(tensors, p + "mix.")
        if spec["type"] == "wkv":
            self.mixer = WkvMixer(p + "wkv", m["heads"], m["dim"], mix, eps, dtype)
        else:
            a, b = m["left"], m["right"]
            left = WindowAttention(p + "left", a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["mask"]["size"], a["scale"],
                                   Rotary(a["rot"]["dims"], a["rot"]["base"], a["rot"].get("scaling")),
                                   Scope(tensors, p + "mix.left."), eps, dtype)
            right = ScaledLinearAttention(p + "right", b["heads"], b["dim"], b["vdim"], b["decay"],
                                          Scope(tensors, p + "mix.right."), eps, dtype)
            self.mixer = ParallelMixer(left, right, m["left_scale"], m["right_scale"])
        self.norm1 = f32(tensors[p + "norm1"])
        self.ff = self.norm2 = None
        if spec.get("mlp") is not None:
            self.ff = GatedFeedForward(Scope(tensors, p + "mlp."))
            self.norm2 = f32(tensors[p + "norm2"])


@register("Sipadra")
class Sipadra(HybridDecoder):
    def __init__(self, config, tensors, dtype=torch.bfloat16):
        self.config, self.dtype = config, dtype
        self.embed = tensors["embed"]
        if tuple(self.embed.shape) != (config.vocab_size, config.n_embd):
            raise ValueError(f"embed is {tuple(self.embed.shape)}, the configuration says {(config.vocab_size, config.n_embd)}")
        self.layers = [_Layer(i, spec, tensors, config.eps, dtype) for i, spec in enumerate(config.layers)]
        self.final_norm = f32(tensors["final.norm"])

    parse = staticmethod(SipadraConfig.from_dict)
    shapes = staticmethod(lambda config: tensor_shapes(config, rank=None))

    @torch.inference_mode()
    def forward(self, idx, targets=None, kv_cache=None, logits_at=None, on_layer=None):
        """fp32 logits (B, T, vocab), or (B, len(logits_at), vocab) at the given places of the T tokens (an
        empty list runs the tokens and returns None).  ``on_layer(i, x)`` sees the stream after each layer."""
        B, T, kv_cache = self.begin(idx, targets, kv_cache)
        cfg = self.config
        with mo.full_precision_sums():
            x = y = w = None
            common = dict(eps=cfg.eps, dtype=self.dtype, B=B, T=T)
            source = dict(tokens=idx.contiguous().view(-1), table=self.embed)
            for i, layer in enumerate(self.layers):
                mixer = layer.mixer
                if mixer.shift is not None:
                    x, _, h = mo.resid_norm(x, y, w, mu=mixer.shift, carry=mixer.carry(kv_cache), **source, **common)
                else:
                    x, h, _ = mo.resid_norm(x, y, w, want_h=True, **source, **common)
                source = {}
                if on_layer is not None and i > 0:
                    on_layer(i - 1, x.clone())
                y, w = mixer(h, kv_cache, B, T), layer.norm1
                if layer.ff is not None:
                    x, h, _ = mo.resid_norm(x, y, w, want_h=True, **common)
                    y, w = layer.ff(h), layer.norm2
            if on_layer is not None:
                on_layer(cfg.n_layer - 1, mo.resid_norm(x.clone(), y, w, want_h=True, **common)[0])
            kv_cache.advance(T)
            n = T
            if logits_at is not None:
                if len(logits_at) == 0:
                    return None
                n = len(logits_at)
                x, y = self.pick(x, B, T, logits_at), self.pick(y, B, T, logits_at)
            _, h, _ = mo.resid_norm(x, y, w, eps=cfg.eps, dtype=self.dtype, B=B, T=n, final_weight=self.final_norm)
            logits = mo.product(h, self.embed, f32_out=True)
            if cfg.logit_softcap is not None:
                mo.softcap(logits, cfg.logit_softcap)
        return logits.view(B, n, -1)

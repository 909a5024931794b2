"""What the decoders that are put together from a list of layers share."""
import torch

from .engine import HybridCache


class Scope:
    """The tensors below a name prefix, looked up without it."""

    def __init__(self, tensors, prefix):
        self.tensors, self.prefix = tensors, prefix

    def __getitem__(self, name):
        return self.tensors[self.prefix + name]


class HybridDecoder:
    """Inference model with GPT's interface: ``config``, ``get_device``, ``make_cache``, ``forward(ids, kv_cache=...)``.

    A design gives ``parse`` (config.json's dict -> configuration), ``shapes`` (the dict -> name -> shape, None for a
    size that the tensors decide), a constructor ``(configuration, tensors, dtype)`` that sets ``embed`` and
    ``layers`` (each with a ``mixer``), and ``forward``."""

    accepts_logits_at = True

    @classmethod
    def from_dict(cls, config, tensors, dtype, device):
        parsed = cls.parse(config)
        for name, shape in cls.shapes(config).items():
            if name not in tensors:
                raise ValueError(f"the weights lack {name}")
            have = tuple(tensors[name].shape)
            if len(have) != len(shape) or any(want not in (None, n) for want, n in zip(shape, have)):
                raise ValueError(f"{name} is {have}, the configuration says {shape}")
        tensors = {k: v.to(device=device, dtype=dtype) for k, v in tensors.items()}
        return cls(parsed, tensors, dtype)

    def get_device(self):
        return self.embed.device

    def make_cache(self, batch_size, seq_len, page_tokens=None, n_pages=None):
        if page_tokens:
            raise NotImplementedError("this model keeps its keys and states in dense rows; page_tokens is not supported")
        cache = HybridCache(batch_size, seq_len, self.get_device())
        for layer in self.layers:
            layer.mixer.declare(cache)
        return cache

    def begin(self, idx, targets, kv_cache):
        """(rows, new tokens, cache) of a forward call."""
        if targets is not None:
            raise NotImplementedError("this model is inference-only")
        B, T = idx.shape
        return B, T, kv_cache if kv_cache is not None else self.make_cache(B, T)

    @staticmethod
    def pick(t, B, T, places):
        """Rows of (B * T, ...) activations at the given places of the T tokens."""
        rows = torch.as_tensor(places, device=t.device)
        return t.view(B, T, *t.shape[1:]).index_select(1, rows).flatten(0, 1).contiguous()

"""Small configurations and helpers shared by the Sipadra tests."""
import torch

from oracle import sipadra_ref as R

YARN = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}


def wkv_layer(heads=3, dim=20, ff=72):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel_layer(heads=4, kv_heads=2, dim=24, vdim=40, window=9, rot_dims=16, base=5000.0, scaling=YARN, scale=0.31, r_heads=3,
                   r_dim=12, r_vdim=28, decay=(0.5, 0.9, 0.995), left_scale=0.7, right_scale=1.3, ff=56):
    return {"type": "parallel", "mlp": {"kind": "dense", "ff": ff} if ff else None, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale,
                 "rot": {"base": base, "dims": rot_dims, "scaling": scaling}},
        "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": list(decay)},
        "left_scale": left_scale, "right_scale": right_scale}}


def config(layers, width=84, vocab=101, eps=3e-5, cap=12.0):
    return {"architecture": "Sipadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


# name -> (configuration, inner width of the decay paths)
CONFIGS = {
    # small heads: padded to the tensor-core kernels; two kinds of layers, one without a feed-forward
    "mixed": (config([parallel_layer(), wkv_layer(), wkv_layer(ff=None), parallel_layer(window=5, decay=(0.8, 0.999, 0.3))]), 7),
    # full-size heads, window across several key tiles, attention group of 5, no frequency scaling
    "wide": (config([wkv_layer(heads=2, dim=64, ff=128), parallel_layer(heads=5, kv_heads=1, dim=128, vdim=128, window=70, rot_dims=64,
                     base=10000.0, scaling=None, scale=128 ** -0.5, r_heads=2, r_dim=64, r_vdim=128, decay=(0.9, 0.99),
                     left_scale=1.0, right_scale=1.0, ff=96)], width=160, vocab=211), 16),
    # sizes that allow no vector accesses, heads beyond the tensor-core kernels, a group of 17, one-token window
    "odd": (config([parallel_layer(heads=2, kv_heads=1, dim=130, vdim=150, window=6, rot_dims=26, r_heads=1, r_dim=9, r_vdim=33,
                    decay=(0.97,), ff=23), wkv_layer(heads=1, dim=37, ff=31),
                    parallel_layer(heads=17, kv_heads=1, dim=6, vdim=5, window=1, rot_dims=6, r_heads=2, r_dim=5, r_vdim=3,
                                   decay=(1.0, 0.6), ff=None)], width=45, vocab=67, cap=5.0), 3),
    # heads above 128 key channels in the recurrences
    "large": (config([wkv_layer(heads=1, dim=136, ff=40), parallel_layer(heads=2, kv_heads=2, dim=32, vdim=64, window=12, rot_dims=32,
                      r_heads=1, r_dim=144, r_vdim=200, decay=(0.98,))], width=64), 5),
}


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def oracle_logits(cfg, weights, toks, **kw):
    return R.forward(cfg, R.widened(weights), toks, **kw)


def build(name, dtype, device="cuda", seed=1):
    """(model, configuration, bf16 weights on the CPU)."""
    from nanochat_b200.sipadra import Sipadra
    cfg, rank = CONFIGS[name]
    weights = R.random_weights(cfg, seed=seed, rank=rank)
    return Sipadra.from_dict(cfg, weights, dtype, torch.device(device)), cfg, weights

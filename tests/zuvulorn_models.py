"""Small configurations and helpers shared by the Zuvulorn tests."""
import torch

from oracle import zuvulorn_ref as R

BANDS = {"factor": 5.0, "low": 1.0, "high": 3.0, "original": 90}


def moe(ff=40, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def rglru(width=72, blocks=3, conv=4, mlp=moe()):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def attention(heads=6, kv_heads=2, dim=24, vdim=40, rot_dims=16, base=3000.0, scaling=BANDS, scale=0.27, kv_from=None, mlp=moe()):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
         "rot": {"base": base, "dims": rot_dims, **({"scaling": scaling} if scaling else {})}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads=4, kv_heads=2, dim=20, vdim=28, conv=4, mlp=moe()):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(layers, width=88, vocab=103, eps=2e-5, streams=3):
    return {"architecture": "Zuvulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers}


# name -> (configuration, inner width of the low-rank paths)
CONFIGS = {
    # small heads padded to the tensor-core kernels, every kind of layer, shared keys twice, layers without experts
    "mixed": (config([delta(), attention(), rglru(mlp=None), attention(kv_from=1, scale=0.4), rglru(width=40, blocks=5, conv=2),
                      attention(kv_from=1, mlp=None)]), 8),
    # full-size heads, one stream, all experts chosen, one key/value head
    "wide": (config([attention(heads=5, kv_heads=1, dim=128, vdim=128, rot_dims=128, base=10000.0, scaling=None, scale=128 ** -0.5,
                               mlp=moe(96, 3, 3)), delta(2, 1, 128, 128, 3, mlp=moe(64, 4, 1)), rglru(192, 1, 4, mlp=moe(128, 8, 2)),
                     delta(3, 3, 64, 128, 4, mlp=None)], width=160, vocab=211, streams=1), 16),
    # sizes that allow no vector accesses, heads beyond the tensor-core kernels, a group of 17
    "odd": (config([attention(heads=2, kv_heads=1, dim=130, vdim=150, rot_dims=26, mlp=moe(23, 3, 1)),
                    delta(3, 1, 37, 33, 2, mlp=moe(31, 7, 3)), rglru(45, 9, 1, mlp=None),
                    attention(heads=17, kv_heads=1, dim=6, vdim=5, rot_dims=6, mlp=moe(9, 2, 2)),
                    attention(heads=17, kv_heads=1, dim=6, vdim=5, rot_dims=6, kv_from=3, mlp=moe(12, 4, 1))],
                   width=45, vocab=67, streams=5), 3),
    # key channels beyond 128, values wider than the single-token kernel, long filters
    "large": (config([delta(1, 1, 200, 136, 9, mlp=moe(48, 6, 1)), delta(2, 2, 150, 64, 4, mlp=None), rglru(64, 2, 16, mlp=moe(16, 2, 1))],
                     width=64, streams=2), 24),
}


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def oracle_logits(cfg, weights, toks, **kw):
    return R.forward(cfg, R.widened(weights), toks, **kw)


def build(name, dtype, device="cuda", seed=1):
    """(model, configuration, bf16 weights on the CPU)."""
    from nanochat_b200.zuvulorn import Zuvulorn
    cfg, rank = CONFIGS[name]
    weights = R.random_weights(cfg, seed=seed, rank=rank)
    return Zuvulorn.from_dict(cfg, weights, dtype, torch.device(device)), cfg, weights

"""Host side of the Zuvulorn design: loading, refusals, rotary bands, what layers keep, and the oracle's own sanity."""
import math

import pytest
import torch

from nanochat_b200 import mixers, models
from nanochat_b200.zuvulorn import Zuvulorn, tensor_shapes
from oracle import zuvulorn_ref as R
from tests.zuvulorn_models import BANDS, CONFIGS, attention, config, delta, moe, oracle_logits, rglru, tokens

CPU = torch.device("cpu")


def test_registry_knows_the_design():
    assert models.architectures()["Zuvulorn"] is Zuvulorn


@pytest.mark.parametrize("name", list(CONFIGS))
def test_loader_checks_names_and_shapes(name):
    cfg, rank = CONFIGS[name]
    w = R.random_weights(cfg, rank=rank)
    assert {k: tuple(v) for k, v in tensor_shapes(cfg, rank).items()} == {k: tuple(v.shape) for k, v in w.items()}
    model = Zuvulorn.from_dict(cfg, w, torch.float32, CPU)
    assert model.config.n_layer == len(cfg["layers"]) and model.config.vocab_size == cfg["vocab"]
    lacking = dict(w)
    del lacking["l0.hc1.mix"]
    with pytest.raises(ValueError, match="l0.hc1.mix"):
        Zuvulorn.from_dict(cfg, lacking, torch.float32, CPU)
    with pytest.raises(ValueError, match="head is"):
        Zuvulorn.from_dict(cfg, {**w, "head": torch.ones(3, 3)}, torch.float32, CPU)


@pytest.mark.parametrize("change,text", [(lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
                                         (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward"),
                                         (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "no keys and values"),
                                         (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "no keys and values"),
                                         (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "no keys and values")])
def test_impossible_layers_are_refused(change, text):
    cfg = config([rglru(mlp=moe()), attention(mlp=moe()), attention(kv_from=1, mlp=moe()), attention(kv_from=1, mlp=moe())])
    change(cfg)
    with pytest.raises(ValueError, match=text):
        Zuvulorn.from_dict(cfg, {}, torch.float32, CPU)


def test_layers_share_keys_and_keep_their_states():
    cfg, rank = CONFIGS["mixed"]
    model = Zuvulorn.from_dict(cfg, R.random_weights(cfg, rank=rank), torch.bfloat16, CPU)
    cache = model.make_cache(2, 50)
    assert list(cache.kv) == ["l1.attention"]
    assert model.layers[3].mixer.source is model.layers[1].mixer and model.layers[5].mixer.source is model.layers[1].mixer
    m, d = cfg["layers"][2]["mixer"], cfg["layers"][0]["mixer"]
    assert cache.state["l2.rglru"].shape == (2, m["width"]) and cache.state["l2.rglru.conv"].shape == (2, m["conv"] - 1, m["width"])
    assert cache.state["l0.channel_delta"].shape == (2, d["heads"], d["dim"], d["vdim"])
    assert cache.state["l0.channel_delta.conv"].shape == (2, d["conv"] - 1, 2 * d["kv_heads"] * d["dim"] + d["heads"] * d["vdim"])
    assert all(t.dtype == torch.float32 for t in cache.state.values())
    with pytest.raises(NotImplementedError):
        model.make_cache(1, 50, page_tokens=192)


@pytest.mark.parametrize("dims,base,scaling", [(16, 3000.0, BANDS), (64, 5e5, {"factor": 4.0, "low": 2.0, "high": 8.0, "original": 700}),
                                               (32, 1e4, None), (8, 40.0, {"factor": 1.0, "low": 1.0, "high": 4.0, "original": 10})])
def test_rotary_table_turns_pairs_like_the_oracle(dims, base, scaling):
    n = 260
    table = mixers.rotary_table(n, dims, base, scaling)
    freqs = R.frequencies(dims, base, scaling)
    x = torch.randn(2, dims + 3, dtype=torch.float64, generator=torch.Generator().manual_seed(dims))
    half = dims // 2
    for pos in (0, 1, 19, n - 1):
        c, s = table[pos, :half].double(), table[pos, half:].double()
        u, v = x[:, :half], x[:, half:dims]
        got = torch.cat([u * c - v * s, v * c + u * s, x[:, dims:]], 1)
        assert torch.allclose(got, R.rotate(x, pos, dims, freqs), atol=2e-6)


def test_the_three_bands():
    scaling = {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 1000}
    turns = torch.tensor([8.0, 4.0, 2.5, 1.0, 0.2], dtype=torch.float64)  # over the original context
    freq = turns * 2 * math.pi / 1000
    got = mixers.banded_scaling(freq, scaling) / freq
    assert torch.allclose(got, torch.tensor([1.0, 1.0, 0.5 + 0.5 / 6, 1 / 6, 1 / 6], dtype=torch.float64))


def test_stacked_products_keep_rows_aligned():
    ws = [torch.randn(n, 6) for n in (5, 8, 2)]
    w, widths = mixers.stacked(ws)
    assert w.shape == (16, 6) and widths == [5, 8, 2] and (w[15:] == 0).all()
    x = torch.randn(3, 6)
    for part, one in zip(mixers.columns(x @ w.t(), widths), ws):
        assert torch.allclose(part, x @ one.t(), atol=1e-6)


def test_oracle_mechanisms_show_in_the_logits():
    """Every tensor moves the oracle's logits, so a comparison with it sees every mechanism."""
    cfg = config([attention(), delta(mlp=None), rglru(), attention(kv_from=0)])
    w = R.random_weights(cfg, seed=5, rank=6)
    toks = tokens(14, cfg["vocab"], 3)
    base = oracle_logits(cfg, w, toks)
    used = set()
    for name in w:
        if ".mlp.e" in name or name in ("final.norm", "embed", "head"):
            continue
        moved = (oracle_logits(cfg, {**w, name: torch.zeros_like(w[name])}, toks) - base).abs().max()
        assert moved > 1e-3, name
    for name in w:
        if ".mlp.e" in name and (oracle_logits(cfg, {**w, name: torch.zeros_like(w[name])}, toks) - base).abs().max() > 1e-4:
            used.add(name.split(".e")[1].split(".")[0])
    assert len(used) >= 4


def test_oracle_sink_and_far_keys():
    T = 12
    q = torch.zeros(T, 1, 2, dtype=torch.float64)
    k, v = torch.zeros(T, 1, 2, dtype=torch.float64), torch.ones(T, 1, 1, dtype=torch.float64)
    out = R.sink_attention(q, k, v, 1.0)[:, 0, 0]  # all scores 0: the sink takes one share of n + 1
    assert torch.allclose(out, torch.arange(1, T + 1).double() / torch.arange(2, T + 2).double())
    q[:, 0, 0], k[0, 0, 0], v[0] = 1.0, 60.0, 5.0
    assert torch.allclose(R.sink_attention(q, k, v, 1.0)[:, 0, 0], torch.full((T,), 5.0, dtype=torch.float64))
    assert R.sink_attention(q, k - 100 * q, v, 1.0)[1:, 0, 0].abs().max() < 1e-15  # the sink takes everything


def test_oracle_delta_rule_overwrites_what_a_key_reads():
    k = torch.zeros(3, 1, 4, dtype=torch.float64)
    k[:, 0, 1] = 1.0
    v = torch.tensor([[[2.0, 3.0]], [[-1.0, 4.0]], [[0.5, 0.25]]], dtype=torch.float64)
    g, one = torch.ones(3, 1, 4, dtype=torch.float64), torch.ones(3, 1, dtype=torch.float64)
    out, _ = R.delta_memory(k, k, v, g, one)
    assert torch.allclose(out, v)  # with beta 1 the newest value replaces the old one
    out, _ = R.delta_memory(k, k, v, g, 0 * one)
    assert (out == 0).all()

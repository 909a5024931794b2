"""Host side of the hybrid design: weight files, registry, rotary tables, caches and the sequence runner."""
import json
import struct

import pytest
import torch

from nanochat_b200 import mixers, models, weights
from nanochat_b200.engine import HybridCache, SequenceRunner
from nanochat_b200.sipadra import Sipadra, tensor_shapes
from oracle import sipadra_ref as R
from tests.sipadra_models import CONFIGS, YARN, config, oracle_logits, parallel_layer, tokens, wkv_layer


def test_safetensors_round_trip_and_bad_files(tmp_path):
    src = {"a": torch.randn(3, 5).bfloat16(), "b.c": torch.arange(7, dtype=torch.int32), "empty": torch.empty(0, 4), "s": torch.tensor(2.5)}
    path = str(tmp_path / "x.safetensors")
    weights.write_safetensors(path, src)
    back = weights.read_safetensors(path)
    assert back.keys() == src.keys()
    for k, v in src.items():
        assert back[k].dtype == v.dtype and back[k].shape == v.shape and torch.equal(back[k], v)
    head = json.dumps({"a": {"dtype": "F32", "shape": [4], "data_offsets": [0, 12]}}).encode()
    (tmp_path / "y").write_bytes(struct.pack("<Q", len(head)) + head + b"\0" * 16)
    with pytest.raises(ValueError, match="data_offsets"):
        weights.read_safetensors(str(tmp_path / "y"))
    (tmp_path / "z").write_bytes(struct.pack("<Q", 1 << 40) + b"{}")
    with pytest.raises(ValueError, match="header"):
        weights.read_safetensors(str(tmp_path / "z"))


def test_registry_knows_both_designs_and_refuses_others(tmp_path):
    found = models.architectures()
    assert found["Sipadra"] is Sipadra and "nanochat" in found
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        models.load_model(str(tmp_path), device="cpu")


def test_registry_loads_a_gpt_folder(tmp_path):
    from nanochat_b200.gpt import GPT, GPTConfig
    cfg = dict(sequence_len=64, vocab_size=64, n_layer=2, n_head=2, n_kv_head=2, n_embd=64)
    ref = GPT(GPTConfig(**cfg))
    ref.init_weights()
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "nanochat", **cfg}))
    weights.write_safetensors(str(tmp_path / "model.safetensors"), {k: v.float() for k, v in ref.state_dict().items()})
    got = models.load_model(str(tmp_path), torch.float32, "cpu")
    assert isinstance(got, GPT) and got.state_dict().keys() == ref.state_dict().keys()
    for k, v in ref.state_dict().items():
        assert torch.equal(got.state_dict()[k], v.float())
    assert got.cos.shape == ref.cos.shape


@pytest.mark.parametrize("name", list(CONFIGS))
def test_loader_checks_names_and_shapes(name):
    cfg, rank = CONFIGS[name]
    w = R.random_weights(cfg, rank=rank)
    assert {k: tuple(v) for k, v in tensor_shapes(cfg, rank).items()} == {k: tuple(v.shape) for k, v in w.items()}
    model = Sipadra.from_dict(cfg, w, torch.float32, torch.device("cpu"))
    assert model.config.n_layer == len(cfg["layers"]) and model.config.vocab_size == cfg["vocab"]
    lacking = dict(w)
    del lacking["final.norm"]
    with pytest.raises(ValueError, match="final.norm"):
        Sipadra.from_dict(cfg, lacking, torch.float32, torch.device("cpu"))
    with pytest.raises(ValueError, match="l0.norm1"):
        Sipadra.from_dict(cfg, {**w, "l0.norm1": torch.ones(3)}, torch.float32, torch.device("cpu"))


def test_unknown_layers_are_refused():
    bad = config([wkv_layer()])
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        Sipadra.from_dict(bad, {}, torch.float32, torch.device("cpu"))
    bad = config([wkv_layer()])
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        Sipadra.from_dict(bad, {}, torch.float32, torch.device("cpu"))


@pytest.mark.parametrize("dims,base,scaling", [(16, 5000.0, YARN), (32, 1e6, {"factor": 2.0, "original": 1024, "fast": 32.0, "slow": 1.0}),
                                               (64, 10000.0, None), (8, 100.0, {"factor": 8.0, "original": 7, "fast": 4.0, "slow": 3.9}),
                                               (6, 50.0, {"factor": 1.0, "original": 4000, "fast": 2.0, "slow": 0.01})])
def test_rotary_table_turns_pairs_like_the_oracle(dims, base, scaling):
    n = 300
    table = mixers.rotary_table(n, dims, base, scaling)
    assert table.shape == (n, dims) and table.dtype == torch.float32
    freqs, amp = R.yarn_frequencies(dims, base, scaling)
    x = torch.randn(2, dims + 3, dtype=torch.float64, generator=torch.Generator().manual_seed(dims))
    half = dims // 2
    for pos in (0, 1, 17, n - 1):
        c, s = table[pos, :half].double(), table[pos, half:].double()
        u, v = x[:, :half], x[:, half:dims]
        got = torch.cat([u * c - v * s, v * c + u * s, x[:, dims:]], 1)
        assert torch.allclose(got, R.rotate(x, pos, dims, freqs, amp), atol=2e-6)


def _cache(batch, cap):
    c = HybridCache(batch, cap, "cpu")
    c.add_kv("a", 2, 4, 6, torch.float32)
    c.add_state("s", (3, 5))
    return c


def test_hybrid_cache_broadcast_rows_and_reset():
    src = _cache(1, 8)
    for t in src.kv["a"]:
        t.normal_()
    src.state["s"].normal_()
    src.advance(5)
    dst = _cache(3, 12)
    dst.prefill(src)
    assert dst.cache_seqlens.tolist() == [5, 5, 5] and dst.get_pos() == 5
    for row in range(3):
        assert torch.equal(dst.kv["a"][0][row, :5], src.kv["a"][0][0, :5]) and torch.equal(dst.state["s"][row], src.state["s"][0])
    with pytest.raises(AssertionError):
        dst.prefill(src)
    other = _cache(1, 9)
    other.kv["a"][1].fill_(7.0)
    other.state["s"].fill_(-1.0)
    other.advance(9)
    dst.load_row(1, other)
    assert dst.cache_seqlens.tolist() == [5, 9, 5] and (dst.kv["a"][1][1, :9] == 7).all() and (dst.state["s"][1] == -1).all()
    assert torch.equal(dst.state["s"][2], src.state["s"][0])
    dst.reset()
    assert dst.cache_seqlens.tolist() == [0, 0, 0] and (dst.state["s"] == 0).all()
    made = []
    dst.add_table("t", lambda n, dev: made.append(n) or torch.zeros(n))
    dst.add_table("t", lambda n, dev: made.append(n) or torch.zeros(n))
    assert made == [12]


class _Counting:
    """Logit 0 of a place is how many tokens its sequence holds by then, logit 1 their sum."""

    def __init__(self):
        self.made = 0

    def get_device(self):
        return torch.device("cpu")

    def make_cache(self, batch, cap, page_tokens=None, n_pages=None):
        self.made += 1
        c = HybridCache(batch, cap, "cpu")
        c.add_state("sum", (1,))
        return c

    def forward(self, ids, kv_cache=None):
        B, T = ids.shape
        total = kv_cache.state["sum"] + ids.float().cumsum(1)
        count = (kv_cache.cache_seqlens[:, None] + torch.arange(1, T + 1)).float()
        kv_cache.state["sum"].copy_(total[:, -1:])
        kv_cache.advance(T)
        return torch.stack([count, total], -1)


def test_sequence_runner_keeps_portions_apart_and_reuses_caches():
    model = _Counting()
    run = SequenceRunner(model, 64)
    assert run.feed("a", [1, 2, 3], [0, 2]).tolist() == [[1, 1], [3, 6]]
    assert run.feed("b", [10], [0]).tolist() == [[1, 10]]
    assert run.feed("a", [4], []) is None
    assert run.feed("a", [5], [0]).tolist() == [[5, 15]]
    run.finish("a")
    run.finish("never seen")
    assert run.feed("c", [2, 2], [1]).tolist() == [[2, 4]] and model.made == 2
    assert run.feed("b", [1], [0]).tolist() == [[2, 11]]


def test_oracle_mechanisms_show_in_the_logits():
    """The oracle's own sanity: every part of a layer moves its output, and the window is as long as it says."""
    cfg = config([parallel_layer(window=4), wkv_layer()])
    w = R.random_weights(cfg, seed=5, rank=6)
    toks = tokens(14, cfg["vocab"], 3)
    base = oracle_logits(cfg, w, toks)
    for name in w:
        if name.endswith(("final.norm", "embed")):
            continue
        moved = oracle_logits(cfg, {**w, name: torch.zeros_like(w[name])}, toks)
        assert (moved - base).abs().max() > 1e-3, name
    q, k, v = torch.zeros(9, 1, 2), torch.zeros(9, 1, 2), torch.zeros(9, 1, 1)
    q[:, :, 0] = 1
    k[3, 0, 0], v[3] = 50.0, 1.0
    out = R.window_attention(q, k, v, 1.0, 4)[:, 0, 0]
    assert (out[3:7] > 0.99).all() and (out[:3] < 1e-6).all() and (out[7:] < 1e-6).all()

"""The whole Zuvulorn model on the GPU against the plain oracle: layers, prompts, portions, decoding, batches, reuse,
greedy generation through Engine, and the command line."""
import json
import os
import struct
import subprocess
import sys

import pytest
import torch

from nanochat_b200 import ops, weights
from nanochat_b200.cli import TokenIds
from nanochat_b200.engine import Engine, SequenceRunner
from oracle import zuvulorn_ref as R
from tests.zuvulorn_models import CONFIGS, attention, build, config, delta, moe, oracle_logits, rglru, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF, F32 = torch.bfloat16, torch.float32
LIMIT = {F32: 3e-5, BF: 0.06}


def ids(toks):
    return torch.tensor([toks], dtype=torch.long, device="cuda")


def position_errors(got, want):
    """Per position: rms of the difference of centred logits, relative to the rms of the oracle's."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    c = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / c.pow(2).mean().sqrt()


def agree(got, want, dtype):
    """All positions within the limit; in bf16 a rounding may turn a token's close second choice of expert, so a few
    positions may differ more."""
    e = position_errors(got, want)
    if dtype == F32:
        return e.max().item() < LIMIT[F32]
    return e.median().item() < LIMIT[BF] / 2 and (e > LIMIT[BF]).double().mean().item() <= 0.08


@pytest.mark.parametrize("name", list(CONFIGS))
def test_layers_and_logits_of_a_prompt(name):
    model, cfg, w = build(name, F32)
    toks = tokens(60, cfg["vocab"])
    want, kept = oracle_logits(cfg, w, toks, keep_layers=True)
    seen = {}
    got = model.forward(ids(toks), on_layer=lambda i, x: seen.__setitem__(i, x))[0]
    for i, x in enumerate(kept):
        assert (seen[i].double().cpu() - x).abs().max() < 2e-5 * x.abs().max(), f"layer {i}"
    assert agree(got, want, F32)
    model, _, _ = build(name, BF)
    assert agree(model.forward(ids(toks))[0], want, BF)
    places = [0, 3, 59]
    some = model.forward(ids(toks), logits_at=places)[0]
    assert some.shape == (3, cfg["vocab"]) and agree(some, want[places], BF)
    assert model.forward(ids(toks), logits_at=[]) is None


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_decoding_agree_with_the_whole(name, dtype):
    model, cfg, w = build(name, dtype)
    n = 150 if name == "wide" else 75
    toks = tokens(n, cfg["vocab"], 3)
    want = oracle_logits(cfg, w, toks)
    whole = model.forward(ids(toks), kv_cache=model.make_cache(1, n))[0]
    assert agree(whole, want, dtype)
    for cuts in ([2, 4, 6, n], [n - 30] + list(range(n - 29, n + 1)), [31, 33, 64, 65, n], list(range(1, n + 1))):
        cache, lo, parts = model.make_cache(1, n), 0, []
        for hi in cuts:
            parts.append(model.forward(ids(toks[lo:hi]), kv_cache=cache)[0])
            lo = hi
        assert cache.get_pos() == n
        assert agree(torch.cat(parts), want, dtype), cuts[:4]
    assert ops.read_status(torch.device("cuda", 0)) == 0


def test_a_long_prompt_takes_the_many_row_kernels():
    """Enough tokens for the tensor-memory experts and the chunked scan; the same tokens in portions do not take them."""
    cfg = config([rglru(64, 2, 3, mlp=moe(56, 3, 2)), attention(mlp=None), delta(2, 1, 32, 64, mlp=moe(72, 2, 1))], width=96, streams=2)
    w = R.random_weights(cfg, seed=4, rank=8)
    toks = tokens(700, cfg["vocab"], 5)
    want = oracle_logits(cfg, w, toks)
    from nanochat_b200.zuvulorn import Zuvulorn
    for dtype in (F32, BF):
        model = Zuvulorn.from_dict(cfg, w, dtype, torch.device("cuda"))
        assert agree(model.forward(ids(toks))[0], want, dtype)
        cache, parts = model.make_cache(1, 700), []
        for lo in range(0, 700, 97):
            parts.append(model.forward(ids(toks[lo:lo + 97]), kv_cache=cache)[0])
        assert agree(torch.cat(parts), want, dtype)


def test_a_long_sequence_decoded_token_by_token():
    model, cfg, w = build("mixed", F32)
    n = 260
    toks = tokens(n, cfg["vocab"], 4)
    want = oracle_logits(cfg, w, toks)
    cache = model.make_cache(1, n)
    got = [model.forward(ids(toks[:20]), kv_cache=cache)[0]] + [model.forward(ids([t]), kv_cache=cache)[0] for t in toks[20:]]
    assert agree(torch.cat(got), want, F32)


@pytest.mark.parametrize("kind", ["attention", "rglru", "channel_delta"])
def test_first_and_far_tokens_reach_the_logits(kind):
    """Changing one early token moves late logits exactly as in the oracle, in a prompt and in decoding."""
    from nanochat_b200.zuvulorn import Zuvulorn
    layer = {"attention": attention(mlp=None), "rglru": rglru(mlp=None), "channel_delta": delta(mlp=None)}[kind]
    cfg = config([layer], width=64)
    w = R.random_weights(cfg, seed=8, rank=4)
    if kind == "rglru":
        w["l0.mix.lam"] = torch.full_like(w["l0.mix.lam"], -12.0)
        w["l0.mix.ra.b"] = torch.full_like(w["l0.mix.ra.b"], -1.0)
        w["l0.mix.o"] = w["l0.mix.o"] * 300
    if kind == "channel_delta":
        w["l0.mix.dt_bias"] = torch.full_like(w["l0.mix.dt_bias"], -12.0)
        w["l0.mix.b"] = w["l0.mix.b"] * 0
    model = Zuvulorn.from_dict(cfg, w, F32, torch.device("cuda"))
    toks = tokens(120, cfg["vocab"], 6)

    def logits(t, decode):
        if not decode:
            return model.forward(ids(t))[0].double().cpu()
        cache = model.make_cache(1, 120)
        return torch.cat([model.forward(ids(t[:40]), kv_cache=cache)[0]] + [model.forward(ids([x]), kv_cache=cache)[0] for x in t[40:]]).double().cpu()

    for place in (0, 1, 60):
        other = list(toks)
        other[place] = (other[place] + 1) % cfg["vocab"]
        want = oracle_logits(cfg, w, other) - oracle_logits(cfg, w, toks)
        assert want[-1].abs().max() > 5e-3
        for decode in (False, True):
            got = logits(other, decode) - logits(toks, decode)
            assert (got - want).abs().max() < 2e-4 + 2e-3 * want[-1].abs().max()
            assert place == 0 or got[:place].abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [F32, BF])
def test_batches_of_unequal_sequences_decode_like_each_alone(dtype):
    model, cfg, w = build("mixed", dtype)
    lengths, steps, cap = [1, 7, 30, 52], 12, 80
    seqs = [tokens(n + steps, cfg["vocab"], 20 + n) for n in lengths]
    batch = model.make_cache(len(lengths), cap)
    for row, (n, s) in enumerate(zip(lengths, seqs)):
        alone = model.make_cache(1, n)
        model.forward(ids(s[:n]), kv_cache=alone)
        batch.load_row(row, alone)
    got = []
    for i in range(steps):
        col = torch.tensor([[s[n + i]] for n, s in zip(lengths, seqs)], dtype=torch.long, device="cuda")
        got.append(model.forward(col, kv_cache=batch))
    got = torch.cat(got, 1)
    want = [oracle_logits(cfg, w, s)[n:] for n, s in zip(lengths, seqs)]
    assert agree(torch.cat(list(got)), torch.cat(want), dtype)
    # a row that is given to another sequence carries nothing over
    s = tokens(9 + steps, cfg["vocab"], 77)
    alone = model.make_cache(1, 9)
    model.forward(ids(s[:9]), kv_cache=alone)
    batch.load_row(2, alone)
    got = []
    for i in range(steps):
        col = torch.tensor([[1], [2], [s[9 + i]], [3]], dtype=torch.long, device="cuda")
        got.append(model.forward(col, kv_cache=batch)[2])
    assert agree(torch.cat(got), oracle_logits(cfg, w, s)[9:], dtype)
    # rows of one length run prompts and portions together too
    two = model.make_cache(3, 40)
    rows = [tokens(40, cfg["vocab"], 90 + i) for i in range(3)]
    both = torch.tensor(rows, dtype=torch.long, device="cuda")
    got = torch.cat([model.forward(both[:, lo:hi], kv_cache=two) for lo, hi in ((0, 25), (25, 27), (27, 40))], 1)
    assert agree(torch.cat(list(got)), torch.cat([oracle_logits(cfg, w, r) for r in rows]), dtype)
    places = model.forward(both[:, :9], kv_cache=model.make_cache(3, 9), logits_at=[8, 2])
    assert agree(torch.cat(list(places)), torch.cat([oracle_logits(cfg, w, r[:9])[[8, 2]] for r in rows]), dtype)


def test_caches_are_used_again_without_a_trace():
    model, cfg, w = build("mixed", BF)
    run = SequenceRunner(model, 90)
    first = tokens(80, cfg["vocab"], 1)
    run.feed("x", first, [79])
    for t in run._live["x"].kv["l1.attention"]:
        t.fill_(float("nan"))
    run.finish("x")
    toks = tokens(50, cfg["vocab"], 2)
    used = torch.cat([run.feed("y", toks[:21], list(range(21))), run.feed("y", toks[21:], list(range(29)))])
    fresh_run = SequenceRunner(model, 90)
    fresh = torch.cat([fresh_run.feed("y", toks[:21], list(range(21))), fresh_run.feed("y", toks[21:], list(range(29)))])
    assert torch.equal(used, fresh)
    assert agree(used, oracle_logits(cfg, w, toks), BF)
    # two live sequences, portions in turn
    a, b = tokens(40, cfg["vocab"], 5), tokens(33, cfg["vocab"], 6)
    out = {"a": [], "b": []}
    for lo in range(0, 40, 10):
        out["a"].append(run.feed("a", a[lo:lo + 10], list(range(10))))
        part = b[lo:lo + 10]
        out["b"].append(run.feed("b", part, list(range(len(part)))))
    for name, toks in (("a", a), ("b", b)):
        assert agree(torch.cat(out[name]), oracle_logits(cfg, w, toks), BF)


# ------------------------------------------------------------------------------------------------
# generation and the command line
# ------------------------------------------------------------------------------------------------
def assert_greedy(cfg, w, prompt, produced, margin):
    """Every produced token is the oracle's argmax, up to candidates closer than `margin`."""
    logits = oracle_logits(cfg, w, prompt + produced)
    for i, tok in enumerate(produced):
        row = logits[len(prompt) - 1 + i]
        assert row.max() - row[tok] <= margin, f"token {i}"


@pytest.mark.parametrize("dtype,margin", [(F32, 1e-3), (BF, 0.5)])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_greedy_generation_through_the_engine(name, dtype, margin):
    model, cfg, w = build(name, dtype)
    prompt = tokens(23, cfg["vocab"], 7)
    graphed, _ = Engine(model, TokenIds()).generate_batch(prompt, num_samples=3, max_tokens=40, temperature=0.0)
    assert len(graphed) == 3 and all(r == graphed[0] and len(r) == 63 for r in graphed)
    assert_greedy(cfg, w, prompt, graphed[0][23:], margin)
    eager, _ = Engine(model, TokenIds(), cuda_graph=False).generate_batch(prompt, num_samples=3, max_tokens=40, temperature=0.0)
    assert eager == graphed
    a, _ = Engine(model, TokenIds()).generate_batch(prompt, num_samples=4, max_tokens=20, temperature=1.0, top_k=20, seed=5)
    b, _ = Engine(model, TokenIds(), cuda_graph=False).generate_batch(prompt, num_samples=4, max_tokens=20, temperature=1.0, top_k=20, seed=5)
    assert a == b and len({tuple(r) for r in a}) > 1
    with pytest.raises(NotImplementedError):
        Engine(model, TokenIds(), page_tokens=192).generate_batch(prompt, max_tokens=2)


def _folder(tmp_path, name):
    cfg, rank = CONFIGS[name]
    w = R.random_weights(cfg, seed=2, rank=rank)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    weights.write_safetensors(str(folder / "model.safetensors"), w)
    return str(folder), cfg, w


def test_generate_command(tmp_path):
    folder, cfg, w = _folder(tmp_path, "mixed")
    prompt = tokens(9, cfg["vocab"], 8)
    out = subprocess.run([sys.executable, "-m", "nanochat_b200.cli", "generate", "--model", folder, "--dtype", "float32", "--tokens",
                          ",".join(map(str, prompt)), "--max-tokens", "24", "--num-samples", "2"], cwd=ROOT, capture_output=True,
                         text=True, timeout=240)
    assert out.returncode == 0, out.stderr[-2000:]
    rows = [[int(t) for t in line.split()] for line in out.stdout.splitlines()]
    assert len(rows) == 2 and rows[0] == rows[1] and len(rows[0]) == 24
    assert_greedy(cfg, w, prompt, rows[0], 1e-3)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run(tmp_path, dtype):
    folder, cfg, w = _folder(tmp_path, "odd")
    a, b = tokens(31, cfg["vocab"], 1), tokens(14, cfg["vocab"], 2)
    steps = [("s", a[:17], [0, 16], []), ("s", a[17:19], [], []), ("s", a[19:30], [3], []), ("s", a[30:], [0], ["s"]), ("t", b, [13, 0], ["t"])]
    text = "".join(json.dumps({"step": i, "entries": [{"id": n, "tokens": t, "want": want}], "end": end}) + "\n"
                   for i, (n, t, want, end) in enumerate(steps))
    out_dir = tmp_path / "out"
    out_dir.mkdir()
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out_dir), "--max-tokens",
                          "40"], input=text, capture_output=True, text=True, timeout=240, cwd=str(tmp_path))
    assert run.returncode == 0, run.stderr[-2000:]
    assert [x for x in run.stdout.splitlines() if x.startswith("done ")] == [f"done {i}" for i in range(5)]
    assert sorted(os.listdir(out_dir)) == ["0.f32", "2.f32", "3.f32", "4.f32"]
    want = {"s": oracle_logits(cfg, w, a), "t": oracle_logits(cfg, w, b)}
    rows, expected = [], []
    for step, name, places in ((0, "s", [0, 16]), (2, "s", [22]), (3, "s", [30]), (4, "t", [13, 0])):
        raw = (out_dir / f"{step}.f32").read_bytes()
        rows.append(torch.tensor(struct.unpack(f"<{len(raw) // 4}f", raw)).view(len(places), cfg["vocab"]))
        expected.append(want[name][places])
    e = position_errors(torch.cat(rows), torch.cat(expected))
    assert e.median() < LIMIT[F32 if dtype == "float32" else BF] and (dtype == "bfloat16" or e.max() < LIMIT[F32])

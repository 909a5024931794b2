"""Each kernel of the Zuvulorn design alone, against the plain oracle in fp64."""
import pytest
import torch

from nanochat_b200 import mixer_ops as mo
from nanochat_b200 import ops
from nanochat_b200.mixers import rotary_table
from oracle import zuvulorn_ref as R
from tests.zuvulorn_models import BANDS

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
TOL = {F32: 3e-5, BF: 1.2e-2}  # relative to the largest value of the result; bf16 rounds inputs and outputs


def rand(*shape, dtype=F32, seed=0, scale=1.0):
    z = torch.randn(*shape, generator=torch.Generator().manual_seed(seed + sum(shape))) * scale
    return z.to(dtype).to(DEV)


def host(t):
    return t.detach().double().cpu()


def close(got, want, dtype=F32, factor=1.0):
    got, want = host(got), host(want)
    assert got.shape == want.shape
    assert torch.isfinite(got).all()
    err, top = (got - want).abs().max().item(), want.abs().max().item()
    assert err <= TOL[dtype] * factor * max(top, 1e-3), f"error {err:.3g} of {top:.3g}"


# ------------------------------------------------------------------------------------------------
# streams
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,S,W,parts", [(1, 1, 84, 1), (15, 3, 45, 2), (2, 2, 1536, 1), (40, 5, 192, 3), (1300, 4, 160, 1),
                                            (3, 2, 9000, 1), (2, 8, 2052, 2)])
def test_hyper_norm(dtype, rows, S, W, parts):
    eps = 3e-4
    x, y = rand(rows, S, W, seed=1), rand(rows, parts, W, dtype=dtype, seed=2)
    mix, out, into, w = rand(S, S, seed=3), rand(S, seed=4), rand(S, seed=5), rand(W, seed=6)
    w_all = {"in": host(into), "mix": host(mix), "out": host(out)}
    new = R.through(list(host(x).unbind(1)), w_all, "", lambda u: host(y).sum(1))
    stream, h = mo.hyper_norm(x.clone(), y, (mix, out), into, w, eps, dtype)
    close(stream, torch.stack(new, 1))
    close(h, R.layer_norm(sum(host(into)[s] * new[s] for s in range(S)), eps, host(w)), dtype)
    keep = x.clone()
    stream, h = mo.hyper_norm(keep, y, (mix, out), None, w, eps, dtype, store=False)
    assert stream is None and torch.equal(keep, x)
    close(h, R.layer_norm(sum(new), eps, host(w)), dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_streams_start_at_the_embedding(dtype):
    V, W, S = 33, 84, 3
    table, into, w = rand(V, W, dtype=dtype), rand(S, seed=1), rand(W, seed=2)
    ids = torch.randint(0, V, (9,), generator=torch.Generator().manual_seed(0)).to(DEV)
    x, h = mo.hyper_norm(None, None, None, into, w, 1e-5, dtype, tokens=ids, table=table, streams=S)
    assert all(torch.equal(x[:, s], table[ids].float()) for s in range(S))
    close(h, R.layer_norm(host(table[ids]) * host(into).sum(), 1e-5, host(w)), dtype)


def test_a_large_common_offset_does_not_hurt_the_norm():
    x, w = rand(4, 1, 256) + 300.0, rand(256, seed=2)
    _, h = mo.hyper_norm(x, None, None, None, w, 1e-5, F32, store=False)
    close(h, R.layer_norm(host(x)[:, 0], 1e-5, host(w)), F32, 2)


# ------------------------------------------------------------------------------------------------
# short convolution
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("C,K", [(40, 4), (33, 3), (256, 2), (5, 1), (12, 7), (520, 16)])
def test_short_conv_in_portions(dtype, C, K):
    B, T = 2, 75
    x = rand(B, T, C + 8, dtype=dtype)  # a column slice of a wider product
    taps, b_in, b = rand(C, K, seed=1), rand(C, seed=2), rand(C, seed=3)
    plain = torch.stack([R.short_conv(host(x[r, :, :C]), host(taps)) for r in range(B)])
    biased = torch.stack([R.short_conv(host(x[r, :, :C]) + host(b_in), host(taps), host(b)) for r in range(B)])
    t = taps.t().contiguous()
    for cuts in ([75], [2, 4, 5, 6, 75], [40, 41, 42, 58, 75], list(range(1, 76))):
        for silu, args, want in ((True, (None, None), R.silu(plain)), (False, (b_in, b), biased)):
            carry, lo, got = torch.zeros(B, K - 1, C, device=DEV), 0, []
            for hi in cuts:
                part = x[:, lo:hi].reshape(-1, C + 8)[:, :C]
                got.append(mo.short_conv(part, t, carry, B, hi - lo, *args, silu=silu).view(B, hi - lo, C))
                lo = hi
            close(torch.cat(got, 1), want, dtype)


# ------------------------------------------------------------------------------------------------
# real-gated recurrence
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("C,blocks", [(72, 3), (45, 9), (64, 1), (1056, 4)])
def test_gated_scan_in_portions(dtype, C, blocks):
    B, T, n = 2, 700 if C == 64 else 90, C // blocks
    u, y = rand(B * T, C, dtype=dtype, seed=1), rand(B * T, C, dtype=dtype, seed=2)
    ra, ri = rand(blocks, n, n, dtype=dtype, seed=3, scale=n ** -0.5), rand(blocks, n, n, dtype=dtype, seed=4, scale=n ** -0.5)
    bias, yb, lam = rand(2, C, seed=5), rand(C, seed=6), rand(C, seed=7) - 3
    want, last = [], []
    for r in range(B):
        uu = host(u).view(B, T, C)[r]
        la, i = R.rglru_gates(uu, host(ra), host(bias[0]).view(blocks, n), host(ri), host(bias[1]).view(blocks, n), host(lam))
        s = R.gated_accumulation(la, i * uu)
        want.append(s * R.gelu_tanh(host(y).view(B, T, C)[r] + host(yb)))
        last.append(s[-1])
    rate = (8 * R.softplus(host(lam))).float().to(DEV)
    w = torch.cat([ra.transpose(1, 2), ri.transpose(1, 2)], 2).contiguous()
    for cuts in ([T], [2, 20, 21, T], [T - 40] + list(range(T - 39, T + 1))):
        state, lo, got = torch.zeros(B, C, device=DEV), 0, []
        for hi in cuts:
            pick = [t.view(B, T, C)[:, lo:hi].reshape(-1, C) for t in (u, y)]
            with mo.full_precision_sums():
                gates = mo.block_product(pick[0], w)
            got.append(mo.gated_scan(*pick, gates, bias, yb, rate, state, B, hi - lo).view(B, hi - lo, C))
            lo = hi
        close(torch.cat(got, 1), torch.stack(want), dtype)
        close(state, torch.stack(last), F32 if dtype == F32 else BF)


def test_gated_scan_remembers_the_first_token():
    T, C = 600, 16
    u = torch.zeros(T, C, device=DEV)
    u[0] = 7.0
    gates = torch.zeros(1, T, 2 * C, device=DEV)
    gates[..., :C] = -20.0  # no decay afterwards; the first token decays everything and writes
    gates[:, 0, :C] = 20.0
    gates[..., C:] = 20.0
    y = torch.full((T, C), 3.0, device=DEV)
    zeros = torch.zeros(2, C, device=DEV)
    out = mo.gated_scan(u, y, gates, zeros, zeros[0], torch.full((C,), 30.0, device=DEV), torch.zeros(1, C, device=DEV), 1, T)
    close(out, torch.full((T, C), 7.0 * R.gelu_tanh(torch.tensor(3.0, dtype=torch.float64)).item()), F32, 2)


# ------------------------------------------------------------------------------------------------
# delta rule
# ------------------------------------------------------------------------------------------------
def delta_case(dtype, B, T, H, G, Dk, Dv, seed=0, strong=False):
    c = {"q": rand(B * T, G * Dk, dtype=dtype, seed=seed), "k": rand(B * T, G * Dk, dtype=dtype, seed=seed + 1),
         "v": rand(B * T, H * Dv, dtype=dtype, seed=seed + 2), "x": rand(B * T, H * Dk, seed=seed + 3) + (25.0 if strong else 0.0),
         "x0": rand(H * Dk, seed=seed + 4) - 1, "rate": torch.exp(rand(H, seed=seed + 5) - 1), "b": rand(B * T, H, dtype=dtype, seed=seed + 6),
         "gate": rand(B * T, H * Dv, dtype=dtype, seed=seed + 7), "norm": rand(Dv, seed=seed + 8)}
    return c


def delta_oracle(c, B, T, H, G, Dk, Dv, eps):
    outs, states = [], []
    group = torch.arange(H) // (H // G)
    for r in range(B):
        f = {n: host(t).view(B, T, -1)[r] for n, t in c.items() if n in "qkvxb" or n == "gate"}
        q = R.unit(f["q"].view(T, G, Dk))[:, group] * Dk ** -0.5
        k = R.unit(f["k"].view(T, G, Dk))[:, group]
        g = torch.exp(-host(c["rate"])[:, None] * R.softplus(f["x"] + host(c["x0"])).view(T, H, Dk))
        o, s = R.delta_memory(q, k, f["v"].view(T, H, Dv), g, torch.sigmoid(f["b"]))
        outs.append((R.rms_norm(o, eps, host(c["norm"])) * torch.sigmoid(f["gate"].view(T, H, Dv))).reshape(T, H * Dv))
        states.append(s)
    return torch.stack(outs), torch.stack(states)


def run_delta(c, B, T, lo, hi, H, G, Dk, Dv, eps, state):
    p = {n: t.view(B, T, -1)[:, lo:hi].reshape(B * (hi - lo), -1) for n, t in c.items() if n in ("q", "k", "v", "x", "b", "gate")}
    out = mo.delta_rule(p["q"], p["k"], p["v"], p["x"], c["x0"], c["rate"], p["b"], state, B, hi - lo, H, G, Dk, Dv, p["gate"],
                        c["norm"], eps)
    return out.view(B, hi - lo, -1)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,G,Dk,Dv", [(4, 2, 20, 28), (2, 2, 64, 64), (3, 1, 37, 33), (2, 1, 128, 128), (1, 1, 200, 136), (2, 2, 96, 24),
                                       (1, 1, 256, 128), (2, 1, 12, 4)])
def test_delta_rule_in_portions(dtype, H, G, Dk, Dv):
    B, T, eps = 2, 43, 2e-4
    c = delta_case(dtype, B, T, H, G, Dk, Dv)
    want, last = delta_oracle(c, B, T, H, G, Dk, Dv, eps)
    for cuts in ([T], [2, 4, 5, 7, 12, T], [T - 20] + list(range(T - 19, T + 1))):
        state, lo, got = torch.zeros(B, H, Dk, Dv, device=DEV), 0, []
        for hi in cuts:
            got.append(run_delta(c, B, T, lo, hi, H, G, Dk, Dv, eps, state))
            lo = hi
        close(torch.cat(got, 1), want, dtype)
        close(state, last, F32, 2)


@pytest.mark.parametrize("B,H,Dk", [(12, 16, 128), (40, 16, 128), (40, 16, 64), (20, 16, 200)])
def test_delta_rule_with_many_heads(B, H, Dk):
    """Enough (row, head) pairs for every arrangement of lanes."""
    T, Dv, eps = 9, 128, 1e-5
    c = delta_case(F32, B, T, H, H, Dk, Dv)
    want, last = delta_oracle(c, B, T, H, H, Dk, Dv, eps)
    state = torch.zeros(B, H, Dk, Dv, device=DEV)
    close(run_delta(c, B, T, 0, T, H, H, Dk, Dv, eps, state), want)
    close(state, last, F32, 2)


def test_strong_decay_neither_overflows_nor_leaks():
    B, T, H, Dk, Dv = 1, 30, 2, 64, 64
    c = delta_case(F32, B, T, H, H, Dk, Dv, strong=True)
    c["rate"] = torch.tensor([9.0, 40.0], device=DEV)
    want, last = delta_oracle(c, B, T, H, H, Dk, Dv, 1e-5)
    state = torch.zeros(B, H, Dk, Dv, device=DEV)
    close(run_delta(c, B, T, 0, T, H, H, Dk, Dv, 1e-5, state), want)
    close(state, last)


def test_a_delta_state_holds_a_far_token():
    """One key written at the start is read back at the end exactly, through hundreds of orthogonal writes."""
    T, D = 500, 64
    k = torch.zeros(T, D, device=DEV)
    k[0, 5] = 1.0
    k[torch.arange(1, T), 6 + torch.arange(1, T) % 50] = 1.0
    q = k.clone()
    q[T - 1] = k[0]
    v = rand(T, D)
    c = {"q": q, "k": k, "v": v, "x": torch.full((T, D), -90.0, device=DEV), "x0": torch.zeros(D, device=DEV),
         "rate": torch.ones(1, device=DEV), "b": torch.full((T, 1), 60.0, device=DEV), "gate": torch.full((T, D), 60.0, device=DEV),
         "norm": torch.ones(D, device=DEV)}
    out = run_delta(c, 1, T, 0, T, 1, 1, D, D, 0.0, torch.zeros(1, 1, D, D, device=DEV))
    close(out[0, -1], R.rms_norm(host(v[0]), 0.0))


# ------------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,G,Dk,Dv,rot", [(6, 2, 24, 40, 16), (4, 4, 128, 128, 128), (3, 1, 37, 9, 6), (2, 1, 64, 80, 0)])
def test_rms_rope_append(dtype, H, G, Dk, Dv, rot):
    B, T, cap, eps, q_scale = 2, 11, 40, 3e-4, 1.7
    x = rand(B * T, (H + G) * Dk + G * Dv + 8, dtype=dtype)
    q, k, v = x[:, :H * Dk], x[:, H * Dk:(H + G) * Dk], x[:, (H + G) * Dk:(H + G) * Dk + G * Dv]
    wq, wk = rand(H * Dk, seed=1), rand(G * Dk, seed=2)
    lens = torch.tensor([0, 23], dtype=torch.int32, device=DEV)
    pad = 128 if max(Dk, Dv) <= 128 else Dk
    kc, vc = (torch.full((B, cap, G, w), 7.0, dtype=dtype, device=DEV) for w in (pad, max(pad, Dv)))
    table = rotary_table(cap, rot, 3000.0, BANDS, DEV) if rot else torch.empty(cap, 0, device=DEV)
    got = mo.rms_rope_append(q, k, v, wq, wk, table, rot, kc, vc, lens, B, T, H, G, Dk, Dv, q_scale, eps)
    only_q = mo.rms_rope_append(q, None, None, wq, None, table, rot, kc.clone(), vc.clone(), lens, B, T, H, G, Dk, Dv, q_scale, eps)
    assert torch.equal(got, only_q)
    freqs = R.frequencies(rot, 3000.0, BANDS)
    for b in range(B):
        L = int(lens[b])
        for t in range(T):
            row = b * T + t
            nq = R.rms_norm(host(q[row]), eps, host(wq)).view(H, Dk)
            nk = R.rms_norm(host(k[row]), eps, host(wk)).view(G, Dk)
            close(got[b, t, :, :Dk], R.rotate(nq, L + t, rot, freqs) * q_scale, dtype)
            close(kc[b, L + t, :, :Dk], R.rotate(nk, L + t, rot, freqs), dtype)
            assert torch.equal(vc[b, L + t, :, :Dv].reshape(-1), v[row])
        assert (got[b, :, :, Dk:] == 0).all() and (kc[b, L:L + T, :, Dk:] == 0).all() and (vc[b, L:L + T, :, Dv:] == 0).all()
        assert (kc[b, L + T:] == 7).all() and (kc[b, :L] == 7).all()
    assert ops.read_status(torch.device("cuda", 0)) == 0


def attend(dtype, q, kc, vc, lens, scale, gate, tensor_cores):
    if tensor_cores:
        return mo.split_p_attention((q.float() * scale * 128 ** 0.5).to(dtype), kc, vc, lens, None, sink=True, gate=gate)
    return mo.window_attention(q, kc, vc, lens, None, scale, sink=True, gate=gate)


@pytest.mark.parametrize("kind", ["tensor cores", "plain bf16", "plain fp32"])
@pytest.mark.parametrize("T", [1, 2, 70, 150])
def test_sink_and_head_gate(kind, T):
    """Scores around the sink's, far above and far below it; a far key that stands out; rows of unequal length."""
    dtype = F32 if kind == "plain fp32" else BF
    B, H, G, D, cap, scale = 4, 4, 2, 128, 520, 2 * 128 ** -0.5  # the factor that the tensor-core form puts on q is exact
    lens = torch.tensor([0, 47, 48, 350], dtype=torch.int32, device=DEV)
    q, kc, vc = (rand(B, n, h, D, dtype=dtype, seed=s) for n, h, s in ((T, H, 1), (cap, G, 2), (cap, G, 3)))
    q[:, :, 0] *= 0.01          # scores near 0: the sink counts like one more key
    if T > 2:
        q[:, 2, 1] = -30 * kc[:, 5, 0]  # all the weight to a few keys
        kc[:, 1] = 3 * q[:, T - 1, ::2]  # one far key for the last token
    gate = rand(B * T, H + 4, dtype=dtype, seed=5)[:, :H]
    got = attend(dtype, q, kc, vc, lens, scale, gate, kind == "tensor cores")
    for b in range(B):
        n = int(lens[b]) + T
        qq = torch.zeros(n, H, D, dtype=torch.float64)
        qq[n - T:] = host(q[b])
        o = R.sink_attention(qq, host(kc[b, :n]), host(vc[b, :n]), scale)[n - T:]
        close(got[b], o * torch.sigmoid(host(gate).view(B, T, H)[b])[:, :, None], dtype, 1.5)
    kc.mul_(0).sub_(q[:, :1, ::2] * 40)  # every score of head 0 and 2 of the first token far below the sink
    got = attend(dtype, q, kc, vc, lens, scale, None, kind == "tensor cores")
    assert torch.isfinite(got).all()
    assert got[:, 0, 2].abs().max() < 1e-6


# ------------------------------------------------------------------------------------------------
# experts
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,E,top", [(1, 8, 1), (3, 5, 5), (64, 64, 6), (256, 16, 4), (33, 30, 3), (9, 300, 8), (700, 7, 2), (4096, 16, 1),
                                        (5000, 40, 3), (3000, 12, 2), (2500, 25, 1), (700, 200, 4), (1200, 1000, 2)])
def test_routing(rows, E, top):
    z = rand(rows, E)
    z[0] = 1.5  # ties go to the lower index
    r = mo.Routing(z, top)
    offsets, slot, scale = r.offsets.cpu(), r.slot.long().cpu(), host(r.scale)
    assert offsets[0] == 0 and offsets[-1] == rows * top and sorted(slot.tolist()) == list(range(rows * top))
    expert = torch.empty(rows * top, dtype=torch.long)
    for e in range(E):
        expert[slot[offsets[e]:offsets[e + 1]]] = e
    expert = expert.view(rows, top)
    assert expert[0].tolist() == list(range(top))
    want = torch.topk(z[1:].cpu(), top, dim=1).indices
    assert torch.equal(expert[1:], want)
    picked = torch.empty(rows * top, dtype=torch.float64)
    picked[slot] = scale
    assert torch.allclose(picked.view(rows, top), torch.sigmoid(host(z).gather(1, expert)), atol=1e-6)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,E,top,W,ff", [(1, 8, 1, 160, 48), (3, 3, 3, 45, 23), (30, 4, 2, 88, 40), (200, 6, 1, 136, 72), (17, 2, 1, 64, 24), (32, 1, 1, 72, 40), (17, 2, 1, 64, 20),
                                             (600, 3, 1, 192, 136), (700, 5, 2, 328, 264), (1500, 4, 1, 64, 512)])
def test_expert_products(dtype, rows, E, top, W, ff):
    h = rand(rows, W, dtype=dtype)
    z = rand(rows, E, seed=1)
    if rows > 100:
        z[:, 0] += 1.0  # unequal loads
    ws = {}
    for e in range(E):
        ws.update({f"e{e}.gate": rand(ff, W, dtype=dtype, seed=2 + e, scale=W ** -0.5), f"e{e}.up": rand(ff, W, dtype=dtype, seed=20 + e, scale=W ** -0.5),
                   f"e{e}.down": rand(W, ff, dtype=dtype, seed=40 + e, scale=ff ** -0.5)})
    w_in = torch.stack([torch.cat([ws[f"e{e}.gate"], ws[f"e{e}.up"]]) for e in range(E)])
    w_down = torch.stack([ws[f"e{e}.down"] for e in range(E)])
    r = mo.Routing(z, top)
    with mo.full_precision_sums():
        y = mo.expert_product(mo.expert_product(h, w_in, r, True), w_down, r, False)
    assert y.shape == (rows, top, W)
    score = torch.sigmoid(host(z))
    chosen = torch.topk(host(z), top, dim=1).indices
    want = torch.zeros(rows, W, dtype=torch.float64)
    for e in range(E):
        mine = (chosen == e).any(1)
        x = host(h)[mine] * score[mine, e:e + 1]
        want[mine] += (R.silu(x @ host(ws[f"e{e}.gate"]).T) * (x @ host(ws[f"e{e}.up"]).T)) @ host(ws[f"e{e}.down"]).T
    close(y.double().sum(1), want, dtype)
    assert ops.read_status(torch.device("cuda", 0)) == 0


def test_an_expert_without_tokens_and_one_with_all():
    rows, E, W, ff = 900, 4, 128, 64
    for dtype in (F32, BF):
        h = rand(rows, W, dtype=dtype)
        z = torch.full((rows, E), -5.0, device=DEV)
        z[:, 2] = 1.0
        w_in, w_down = rand(E, 2 * ff, W, dtype=dtype, scale=W ** -0.5), rand(E, W, ff, dtype=dtype, scale=ff ** -0.5)
        r = mo.Routing(z, 1)
        assert r.offsets.tolist() == [0, 0, 0, rows, rows]
        y = mo.expert_product(mo.expert_product(h, w_in, r, True), w_down, r, False)[:, 0]
        x = host(h) * torch.sigmoid(torch.tensor(1.0, dtype=torch.float64))
        want = (R.silu(x @ host(w_in[2, :ff]).T) * (x @ host(w_in[2, ff:]).T)) @ host(w_down[2]).T
        close(y, want, dtype)

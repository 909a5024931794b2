"""Each kernel of the hybrid design alone, against the plain oracle in fp64."""
import pytest
import torch

from nanochat_b200 import mixer_ops as mo
from nanochat_b200.mixers import rotary_table
from oracle import sipadra_ref as R
from tests.sipadra_models import YARN

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
TOL = {F32: 3e-5, BF: 1.2e-2}  # relative to the largest value of the result; bf16 rounds inputs and outputs


def rand(*shape, dtype=F32, seed=0, scale=1.0):
    z = torch.randn(*shape, generator=torch.Generator().manual_seed(seed + sum(shape))) * scale
    return z.to(dtype).to(DEV)


def close(got, want, dtype=F32, factor=1.0):
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape
    assert torch.isfinite(got).all()
    err, top = (got - want).abs().max().item(), want.abs().max().item()
    assert err <= TOL[dtype] * factor * max(top, 1e-3), f"error {err:.3g} of {top:.3g}"


def host(t):
    return t.detach().double().cpu()


# ------------------------------------------------------------------------------------------------
# elementwise steps
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("B,T,W", [(1, 1, 84), (3, 5, 45), (2, 1, 1536), (1, 40, 192), (2, 1400, 160), (1, 3, 8192)])
def test_resid_norm(dtype, B, T, W):
    eps, rows = 3e-4, B * T
    x, y, w = rand(rows, W, seed=1), rand(rows, W, dtype=dtype, seed=2), rand(W, seed=3)
    fw, mu, carry = rand(W, seed=4), rand(5, W, seed=5), rand(B, W, seed=6)
    stream = host(x) + R.rms_norm(host(y), eps, host(w))
    new, h, _ = mo.resid_norm(x.clone(), y, w, eps, dtype, B, T, want_h=True)
    close(new, stream)
    close(h, stream, dtype)
    _, h, _ = mo.resid_norm(x.clone(), y, w, eps, dtype, B, T, final_weight=fw)
    close(h, R.rms_norm(stream, eps, host(fw)), dtype)
    # token shift: the row before, or the carried vector for the first token of the call
    old, moved = carry.clone(), carry.clone()
    new, h, mix = mo.resid_norm(x, y, w, eps, dtype, B, T, mu=mu, carry=moved)
    assert h is None
    close(new, stream)
    cur = stream.view(B, T, W)
    before = torch.cat([host(old)[:, None], cur[:, :-1]], 1)
    for m in range(5):
        close(mix[m], (cur + (before - cur) * host(mu[m])).view(rows, W), dtype)
    assert torch.equal(moved, new.view(B, T, W)[:, -1])
    if dtype == BF:  # an fp32 sublayer output
        new, _, _ = mo.resid_norm(x.clone(), y.float(), w, eps, dtype, B, T, want_h=True)
        close(new, stream)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_start_of_the_trunk(dtype):
    B, T, W, V = 2, 7, 84, 33
    table, mu = rand(V, W, dtype=dtype), rand(5, W, seed=9)
    ids = torch.randint(0, V, (B * T,), generator=torch.Generator().manual_seed(0)).to(DEV)
    carry = torch.zeros(B, W, device=DEV)
    x, _, mix = mo.resid_norm(None, None, None, 1e-6, dtype, B, T, tokens=ids, table=table, mu=mu, carry=carry)
    assert torch.equal(x, table[ids].float())
    cur = host(x).view(B, T, W)
    before = torch.stack([R.token_shift(c) for c in cur])
    close(mix[3], (cur + (before - cur) * host(mu[3])).view(B * T, W), dtype)
    x, h, _ = mo.resid_norm(None, None, None, 1e-6, dtype, B, T, tokens=ids, table=table, want_h=True)
    assert torch.equal(h, table[ids])


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,F", [(1, 23), (3, 72), (70, 384), (2, 5504)])
def test_silu_mul(dtype, rows, F):
    gu = rand(rows, 2 * F, dtype=dtype, scale=3.0)
    close(mo.silu_mul(gu), R.silu(host(gu[:, :F])) * host(gu[:, F:]), dtype)


def test_tanh_split_and_softcap():
    z = rand(37, 19, scale=2.0)
    close(mo.tanh_split(z, F32), torch.tanh(host(z)))
    two = mo.tanh_split(z, BF)
    assert two.shape == (37, 38)
    err = (host(two[:, :19]) + host(two[:, 19:]) - torch.tanh(host(z))).abs().max()
    assert err < 2.0 ** -16  # two bf16 terms keep 16 bits; one alone is off by up to 2^-9
    logits = rand(5, 1237, scale=40.0)
    want = 7.0 * torch.tanh(host(logits) / 7.0)
    close(mo.softcap(logits, 7.0), want)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("silu_gate", [False, True])
@pytest.mark.parametrize("rows,C,group", [(3, 99, 33), (5, 256, 256), (2, 2048, 2048), (4, 272, 136), (1, 12, 12)])
def test_gated_norm(dtype, silu_gate, rows, C, group):
    wide = rand(rows, C + 8, dtype=dtype, seed=3)
    x, gate, w = rand(rows, C, seed=1), wide[:, 8:], rand(C, seed=2)
    g = host(gate)
    want = R.rms_norm(host(x).view(rows, -1, group), 2e-5).view(rows, C) * host(w) * (R.silu(g) if silu_gate else torch.sigmoid(g))
    close(mo.gated_norm(x, gate, w, group, 2e-5, silu_gate), want, dtype)


# ------------------------------------------------------------------------------------------------
# rotation, unit norm, append
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,G,dim,vdim,rot,pad", [(4, 2, 24, 40, 16, 128), (6, 1, 128, 128, 128, 128), (3, 3, 7, 5, 6, 7), (2, 1, 130, 150, 26, 150)])
def test_rope_unit_append(dtype, H, G, dim, vdim, rot, pad):
    B, T, cap, eps = 2, 5, 40, 1e-4
    kw, vw = max(pad, dim), max(pad, vdim)
    rows = rand(B * T, (H + G) * dim + G * vdim + 3, dtype=dtype)
    q, k, v = rows[:, :H * dim], rows[:, H * dim:(H + G) * dim], rows[:, (H + G) * dim:(H + G) * dim + G * vdim]
    kc = torch.full((B, cap, G, kw), 9.0, dtype=dtype, device=DEV)
    vc = torch.full((B, cap, G, vw), 9.0, dtype=dtype, device=DEV)
    lens = torch.tensor([0, 33], dtype=torch.int32, device=DEV)
    table = rotary_table(cap, rot, 5000.0, YARN, DEV)
    got = mo.rope_unit_append(q, k, v, table, rot, kc, vc, lens, B, T, H, G, dim, vdim, 0.7, eps)
    freqs, amp = R.yarn_frequencies(rot, 5000.0, YARN)
    for b in range(B):
        for t in range(T):
            pos, row = int(lens[b]) + t, b * T + t
            for what, src, n, scale in ((got[b, t], q, H, 0.7), (kc[b, pos], k, G, 1.0)):
                want = R.rms_norm(R.rotate(host(src[row]).view(n, dim), pos, rot, freqs, amp), eps) * scale
                close(what[:, :dim], want, dtype)
                assert (what[:, dim:] == 0).all()
            assert torch.equal(vc[b, pos, :, :vdim], v[row].view(G, vdim)) and (vc[b, pos, :, vdim:] == 0).all()
    untouched = [(0, T, cap), (1, 0, 33), (1, 33 + T, cap)]
    assert all((kc[b, lo:hi] == 9).all() and (vc[b, lo:hi] == 9).all() for b, lo, hi in untouched)


def test_append_beyond_the_capacity_is_flagged():
    from nanochat_b200 import ops
    kc, vc = (torch.zeros(1, 8, 1, 128, dtype=BF, device=DEV) for _ in range(2))
    lens = torch.tensor([6], dtype=torch.int32, device=DEV)
    q = rand(4, 128, dtype=BF)
    ops.read_status(DEV)
    mo.rope_unit_append(q, q, q, rotary_table(8, 32, 100.0, None, DEV), 32, kc, vc, lens, 1, 4, 1, 1, 128, 128, 1.0, 1e-6)
    assert ops.read_status(DEV) & 1
    assert (kc[0, 6:] != 0).any() and (kc[0, :6] == 0).all()


# ------------------------------------------------------------------------------------------------
# windowed attention: both kernels, prompts, portions and single tokens
# ------------------------------------------------------------------------------------------------
def _attend(kind, q, kc, vc, lens, window, scale):
    if kind == "split_p":
        return mo.split_p_attention(q, kc, vc, lens, window)
    return mo.window_attention(q, kc, vc, lens, window, scale)


def _caches(k, v, dtype, cap):
    T = k.shape[0]
    kc = torch.full((1, cap, *k.shape[1:]), float("nan"), dtype=dtype, device=DEV)  # stale rows must not be read
    vc = torch.full((1, cap, *v.shape[1:]), float("nan"), dtype=dtype, device=DEV)
    kc[0, :T], vc[0, :T] = k, v
    return kc, vc


ATTN = [("split_p", BF, 6, 1, 128, 128), ("split_p", BF, 4, 4, 128, 128), ("split_p", BF, 12, 1, 128, 128), ("any", F32, 6, 2, 24, 40),
        ("any", BF, 17, 1, 6, 5), ("any", F32, 2, 1, 200, 260), ("any", F32, 3, 3, 128, 128)]


@pytest.mark.parametrize("kind,dtype,H,G,dim,vdim", ATTN)
@pytest.mark.parametrize("window", [1, 2, 48, 49, 64, 129, 5000])
def test_window_attention_in_portions(kind, dtype, H, G, dim, vdim, window):
    T = 150
    scale = 128 ** -0.5 if kind == "split_p" else 0.4 * dim ** -0.5
    q, k, v = rand(T, H, dim, dtype=dtype, seed=1, scale=2.0), rand(T, G, dim, dtype=dtype, seed=2, scale=2.0), rand(T, G, vdim, dtype=dtype, seed=3)
    want = R.window_attention(host(q), host(k), host(v), scale, window)
    for cuts in ([T], [64, 65, 80, 82, 83, T], [1, 2, 48, 49, 50, 129, 130, T]):
        at = 0
        for hi in cuts:
            kc, vc = _caches(k[:hi], v[:hi], dtype, T + 9)
            lens = torch.tensor([at], dtype=torch.int32, device=DEV)
            got = _attend(kind, q[None, at:hi].contiguous(), kc, vc, lens, window, scale)
            close(got[0], want[at:hi], dtype, 0.5)
            at = hi


@pytest.mark.parametrize("kind,dtype,H,G,dim,vdim", ATTN[:5])
@pytest.mark.parametrize("window", [5, 48, 64, 200])
def test_one_key_that_stands_out_is_seen_just_inside_the_window_only(kind, dtype, H, G, dim, vdim, window):
    T, far = 300, 37
    scale = 128 ** -0.5 if kind == "split_p" else 1.0
    q, k, v = torch.zeros(T, H, dim), torch.zeros(T, G, dim), torch.zeros(T, G, vdim)
    q[:, :, 0], k[far, :, 0], v[far] = 1.0, 20.0 / scale, 1.0  # its score is 20, all others 0
    q, k, v = (t.to(dtype).to(DEV) for t in (q, k, v))
    kc, vc = _caches(k, v, dtype, T)
    out = _attend(kind, q[None].contiguous(), kc, vc, torch.zeros(1, dtype=torch.int32, device=DEV), window, scale)[0].float()
    assert (out[:far].abs() < 1e-6).all() and (out[far:far + window] > 0.999).all() and (out[far + window:].abs() < 1e-6).all()
    for pos in (far - 1, far, far + window - 1, far + window):  # the same by decoding
        one = _attend(kind, q[None, pos:pos + 1].contiguous(), kc, vc, torch.tensor([pos], dtype=torch.int32, device=DEV), window, scale)
        assert torch.allclose(one[0, 0].float(), out[pos], atol=1e-3)


def test_probabilities_keep_their_low_bits():
    """Two values of opposite sign under nearly equal weights: with weights rounded to bf16 the difference is lost."""
    T, H = 64, 4
    q, k, v = torch.zeros(1, 1, H, 128), torch.zeros(T, 1, 128), torch.zeros(T, 1, 128)
    q[..., 0] = 1.0
    k[::2, 0, 0] = 128 ** 0.5 * 0.0015  # scores 0.0015 and 0: weights differ by 1 part in 670
    v[::2], v[1::2] = 1.0, -1.0
    kc, vc = _caches(k.to(BF).to(DEV), v.to(BF).to(DEV), BF, T)
    want = R.window_attention(torch.cat([torch.zeros(T - 1, H, 128).double(), q[0].double()]), host(kc[0]), host(vc[0]), 128 ** -0.5, T)[-1]
    lens = torch.tensor([T - 1], dtype=torch.int32, device=DEV)
    got = mo.split_p_attention(q.to(BF).to(DEV), kc, vc, lens, T)
    close(got[0, 0], want, BF)
    two = mo.split_p_attention(q.to(BF).to(DEV).expand(1, 2, H, 128).contiguous(), kc, vc, lens - 1, T)
    close(two[0, 1], want, BF)


def test_rows_of_unequal_length_attend_like_each_alone():
    H, G, window, cap = 6, 2, 70, 400
    lens_l = [0, 5, 69, 70, 71, 333]
    kc, vc = rand(6, cap, G, 128, dtype=BF, seed=4), rand(6, cap, G, 128, dtype=BF, seed=5)
    for T in (1, 3):
        q = rand(6, T, H, 128, dtype=BF, seed=6)
        lens = torch.tensor(lens_l, dtype=torch.int32, device=DEV)
        both = mo.split_p_attention(q, kc, vc, lens, window)
        for b in range(6):
            alone = mo.split_p_attention(q[b:b + 1].contiguous(), kc[b:b + 1], vc[b:b + 1], lens[b:b + 1], window)
            assert torch.allclose(both[b].float(), alone[0].float(), atol=4e-3)


# ------------------------------------------------------------------------------------------------
# recurrences
# ------------------------------------------------------------------------------------------------
class Wkv:
    def __init__(self, B, T, H, D, dtype, seed=0):
        n, HD = B * T, H * D
        self.B, self.T, self.H, self.D, self.dtype = B, T, H, D, dtype
        self.r, self.k, self.v, self.g = (rand(n, HD, dtype=dtype, seed=seed + i) for i in range(4))
        self.x = rand(n, HD, seed=seed + 5) * 0.7
        self.x0, self.u, self.w = rand(HD, seed=seed + 6) * 1.5 - 2, rand(HD, seed=seed + 7), rand(HD, seed=seed + 8)

    def run(self, state, lo=0, hi=None, gated=True):
        hi = self.T if hi is None else hi
        cut = lambda t: t.view(self.B, self.T, -1)[:, lo:hi].reshape(self.B * (hi - lo), -1).contiguous()
        extra = dict(gate=cut(self.g), norm_weight=self.w, eps=1e-5) if gated else {}
        return mo.recurrent(cut(self.r), cut(self.k), cut(self.v), state, self.B, hi - lo, self.H, self.D, self.D,
                            decay_logits=cut(self.x), decay_bias=self.x0, bonus=self.u, **extra).view(self.B, hi - lo, -1)

    def oracle(self, b, gated=True):
        T, H, D = self.T, self.H, self.D
        rows = lambda t: host(t).view(self.B, T, H, D)[b]
        w = torch.exp(-torch.exp(rows(self.x) + host(self.x0).view(H, D)))
        o, state = R.wkv_memory(rows(self.r), rows(self.k), rows(self.v), w, host(self.u).view(H, D))
        if gated:
            o = R.rms_norm(o, 1e-5) * host(self.w).view(H, D) * R.silu(rows(self.g))
        return o.reshape(T, H * D), state


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("B,T,H,D", [(1, 1, 3, 20), (2, 1, 2, 64), (3, 1, 1, 128), (2, 2, 2, 48), (1, 37, 3, 20), (2, 16, 2, 64), (1, 17, 1, 37),
                                     (2, 33, 2, 32), (1, 50, 2, 128), (1, 5, 2, 9), (1, 1, 1, 37)])
def test_wkv_recurrence(dtype, B, T, H, D):
    c = Wkv(B, T, H, D, dtype)
    state = torch.zeros(B, H, D, D, device=DEV)
    got = c.run(state)
    for b in range(B):
        want, end = c.oracle(b)
        close(got[b], want, dtype)
        close(state[b], end)


@pytest.mark.parametrize("D", [136, 160, 256])
def test_wkv_recurrence_with_wide_heads_is_left_ungated(D):
    c = Wkv(1, 21, 1, D, F32)
    state = torch.zeros(1, 1, D, D, device=DEV)
    got = c.run(state, gated=False)
    assert got.dtype == F32
    want, end = c.oracle(0, gated=False)
    close(got[0], want)
    close(state[0], end)
    one = c.run(state.clone(), 20, 21, gated=False)
    assert torch.isfinite(one).all()


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,D", [(2, 64), (3, 20), (1, 37)])
def test_wkv_state_has_the_same_bits_however_the_tokens_are_cut(dtype, H, D):
    T = 61
    c = Wkv(2, T, H, D, dtype, seed=30)
    whole_state = torch.zeros(2, H, D, D, device=DEV)
    whole = c.run(whole_state)
    for cuts in ([2, 4, 6, 59, 61], [16, 17, 33, 61], [1, 5, 6, 7, 61], list(range(1, T + 1))):
        state, parts, lo = torch.zeros_like(whole_state), [], 0
        for hi in cuts:
            parts.append(c.run(state, lo, hi))
            lo = hi
        assert torch.allclose(torch.cat(parts, 1).float(), whole.float(), rtol=2e-2 if dtype == BF else 1e-4, atol=2e-2 if dtype == BF else 1e-5)
        assert torch.allclose(state, whole_state, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("B,T,H,D", [(1, 700, 2, 64), (1, 1025, 1, 20), (2, 640, 3, 128)])
def test_wkv_long_prompts_in_segments(B, T, H, D):
    from nanochat_b200 import _lib
    assert _lib.lib.nckv_recurrent_workspace_bytes(B, T, H, D, D) > 0  # this shape is cut into segments
    c = Wkv(B, T, H, D, F32, seed=50)
    start = rand(B, H, D, D, seed=77)
    state = start.clone()
    got = c.run(state)
    again, lo, parts = start.clone(), 0, []
    for hi in (T // 3, T // 3 + 2, T):
        parts.append(c.run(again, lo, hi))
        lo = hi
    close(torch.cat(parts, 1), got)
    close(again, state)
    zero = torch.zeros(B, H, D, D, device=DEV)
    close(c.run(zero)[B - 1], c.oracle(B - 1)[0])
    close(zero[B - 1], c.oracle(B - 1)[1])


def test_wkv_remembers_and_forgets_far_tokens():
    """A loud first token under slow decay is still heard hundreds of tokens later; channels that decay at once forget it."""
    T, H, D = 400, 1, 32
    c = Wkv(1, T, H, D, F32, seed=9)
    c.x.zero_()
    c.x0[:16], c.x0[16:] = -12.0, 3.0  # w = exp(-6e-6) and exp(-20)
    c.k.mul_(0.01)
    c.k[0] = 30.0
    state = torch.zeros(1, H, D, D, device=DEV)
    got, want = c.run(state, gated=False), c.oracle(0, gated=False)[0]
    close(got[0], want)
    far = state[0, 0]
    assert far[:16].abs().mean() > 10 and far[16:].abs().max() < 1.0
    quiet = Wkv(1, T, H, D, F32, seed=9)
    assert not torch.allclose(quiet.run(torch.zeros_like(state), gated=False), got)


def test_strong_decay_stays_finite():
    c = Wkv(1, 40, 2, 48, BF, seed=3)
    c.x.mul_(10.0)
    c.x0.fill_(6.0)  # exp(-exp(.)) underflows to 0 for most channels
    state = torch.zeros(1, 2, 48, 48, device=DEV)
    close(c.run(state)[0], c.oracle(0)[0], BF)
    close(state[0], c.oracle(0)[1])


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("B,T,H,dim,vdim", [(1, 1, 3, 12, 28), (3, 1, 2, 128, 256), (2, 40, 3, 12, 28), (1, 33, 2, 64, 128), (1, 21, 1, 144, 200),
                                            (2, 19, 1, 9, 33), (1, 1, 2, 5, 3), (1, 900, 2, 64, 72), (2, 2, 2, 128, 128)])
def test_scaled_linear_attention(dtype, B, T, H, dim, vdim):
    rows = rand(B * T, H * (2 * dim + vdim) + 8, dtype=dtype, seed=2)
    q, k, v = rows[:, 8:].split([H * dim, H * dim, H * vdim], 1)
    decay = [1.0, 0.3, 0.98][:H]
    state = torch.zeros(B, H, dim, vdim, device=DEV)
    args = dict(decay=torch.tensor(decay, device=DEV), silu_inputs=True)
    got = mo.recurrent(q, k, v, state, B, T, H, dim, vdim, **args).view(B, T, H, vdim)
    ends = []
    for b in range(B):
        part = lambda t, d: R.silu(host(t).view(B, T, H, d)[b])
        want, end = R.decaying_memory(part(q, dim), part(k, dim), part(v, vdim), decay)
        close(got[b], want, F32, 2.0)
        close(state[b], end, F32, 2.0)
        ends.append(end)
    if B == 1 and T > 2:  # in portions
        again, lo = torch.zeros_like(state), 0
        for hi in (2, 3, T // 2, T):
            mo.recurrent(q[lo:hi], k[lo:hi], v[lo:hi], again, 1, hi - lo, H, dim, vdim, **args)
            lo = hi
        close(again[0], ends[0], F32, 2.0)

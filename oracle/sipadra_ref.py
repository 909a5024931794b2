"""Plain, slow restatement of the Sipadra decoder in torch on the CPU.  TEST INFRASTRUCTURE ONLY.

One function per mechanism, whole sequences, one token after the other where the mechanism is a
recurrence, in the dtype of the weights it is given (float64 in the tests).  Shares no code with the
product: no cache, no state manager, no fused step.
"""
import math

import torch


# ------------------------------------------------------------------------------------------------
# mechanisms
# ------------------------------------------------------------------------------------------------
def rms_norm(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def silu(z):
    return z * torch.sigmoid(z)


def yarn_frequencies(dims, base, scaling=None):
    """(angular frequency per pair as a list, factor on cos and sin)."""
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freqs, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def pair_of(turns):  # (real-valued) index of the pair that makes `turns` turns over the original context
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, position, dims, freqs, amplitude):
    """x: (heads, dim) of one token; the first `dims` channels turn, pair (i, i + dims / 2)."""
    half = dims // 2
    angle = torch.tensor([position * f for f in freqs], dtype=torch.float64)
    c = (torch.cos(angle) * amplitude).to(x.dtype)
    s = (torch.sin(angle) * amplitude).to(x.dtype)
    u, v, rest = x[:, :half], x[:, half:dims], x[:, dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], 1)


def window_attention(q, k, v, scale, window):
    """q: (T, H, d), k: (T, G, d), v: (T, G, e): softmax over the `window` latest keys, itself included."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        first = max(0, i - window + 1)
        for h in range(H):
            g = h // (H // G)
            score = (k[first:i + 1, g] @ q[i, h]) * scale
            out[i, h] = torch.softmax(score, 0) @ v[first:i + 1, g]
    return out


def decaying_memory(q, k, v, decay):
    """q, k: (T, H, d), v: (T, H, e), decay: H numbers.  S <- decay S + k v^T, then o = S^T q."""
    T, H, d = q.shape
    state = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    decay = torch.tensor(decay, dtype=torch.float64).to(q.dtype)
    out = []
    for t in range(T):
        state = decay[:, None, None] * state + torch.einsum("hd,he->hde", k[t], v[t])
        out.append(torch.einsum("hde,hd->he", state, q[t]))
    return torch.stack(out), state


def wkv_memory(r, k, v, w, u):
    """r, k, v, w: (T, H, d), u: (H, d).  o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T."""
    T, H, d = r.shape
    state = torch.zeros(H, d, v.shape[2], dtype=r.dtype)
    out = []
    for t in range(T):
        kv = torch.einsum("hd,he->hde", k[t], v[t])
        out.append(torch.einsum("hde,hd->he", state + u[:, :, None] * kv, r[t]))
        state = w[t][:, :, None] * state + kv
    return torch.stack(out), state


def token_shift(h):
    """The previous token's row; zeros before the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


# ------------------------------------------------------------------------------------------------
# mixers, feed-forward, model
# ------------------------------------------------------------------------------------------------
def left_mixer(w, pre, h, cfg, eps):
    T = h.shape[0]
    H, G, d, e = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, d)
    k = (h @ w[pre + "k"].T).view(T, G, d)
    v = (h @ w[pre + "v"].T).view(T, G, e)
    rot = cfg["rot"]
    freqs, amp = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q = torch.stack([rotate(q[t], t, rot["dims"], freqs, amp) for t in range(T)])
    k = torch.stack([rotate(k[t], t, rot["dims"], freqs, amp) for t in range(T)])
    q, k = rms_norm(q, eps), rms_norm(k, eps)
    o = window_attention(q, k, v, cfg["scale"], cfg["mask"]["size"])
    return o.reshape(T, H * e) @ w[pre + "o"].T


def right_mixer(w, pre, h, cfg, eps):
    T = h.shape[0]
    H, d, e = cfg["heads"], cfg["dim"], cfg["vdim"]
    q = silu(h @ w[pre + "q"].T).view(T, H, d)
    k = silu(h @ w[pre + "k"].T).view(T, H, d)
    v = silu(h @ w[pre + "v"].T).view(T, H, e)
    o, _ = decaying_memory(q, k, v, cfg["decay"])
    o = rms_norm(o.reshape(T, H * e), eps, w[pre + "norm"]) * torch.sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def parallel_mixer(w, pre, h, cfg, eps):
    return (cfg["left_scale"] * left_mixer(w, pre + "left.", h, cfg["left"], eps)
            + cfg["right_scale"] * right_mixer(w, pre + "right.", h, cfg["right"], eps))


def wkv_mixer(w, pre, h, cfg, eps):
    T = h.shape[0]
    H, d = cfg["heads"], cfg["dim"]
    before = token_shift(h)
    mix = {s: h + (before - h) * w[pre + "mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[pre + s].T).view(T, H, d) for s in "rkv")
    gate = silu(mix["g"] @ w[pre + "g"].T)
    low = torch.tanh(mix["w"] @ w[pre + "w1"].T) @ w[pre + "w2"].T + w[pre + "w0"]
    decay = torch.exp(-torch.exp(low)).view(T, H, d)
    o, _ = wkv_memory(r, k, v, decay, w[pre + "u"])
    o = rms_norm(o, eps).reshape(T, H * d) * w[pre + "norm"] * gate
    return o @ w[pre + "o"].T


def dense_ff(w, pre, h):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


MIXERS = {"parallel": parallel_mixer, "wkv": wkv_mixer}


def forward(config, weights, tokens, keep_layers=False):
    """Logits (T, vocab) of one sequence; with keep_layers also the residual stream after every layer."""
    eps = config["norm"]["eps"]
    w = weights
    x = w["embed"][torch.as_tensor(tokens)]
    kept = []
    for i, layer in enumerate(config["layers"]):
        pre = f"l{i}."
        y = MIXERS[layer["type"]](w, pre + "mix.", x, layer["mixer"], eps)
        x = x + rms_norm(y, eps, w[pre + "norm1"])
        if layer.get("mlp") is not None:
            x = x + rms_norm(dense_ff(w, pre + "mlp.", x), eps, w[pre + "norm2"])
        kept.append(x)
    logits = rms_norm(x, eps, w["final.norm"]) @ w["embed"].T
    cap = config["logit_softcap"]
    logits = cap * torch.tanh(logits / cap)
    return (logits, kept) if keep_layers else logits


# ------------------------------------------------------------------------------------------------
# small models for tests
# ------------------------------------------------------------------------------------------------
def tensor_shapes(config, rank=8):
    """name -> shape of every tensor a configuration needs; `rank` is the inner width of the decay path."""
    W, V = config["width"], config["vocab"]
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        out[p + "norm1"] = (W,)
        if layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                out[p + "mix.mu." + s] = (W,)
            for s in "rkvg":
                out[p + "mix." + s] = (n, W)
            out.update({p + "mix.w1": (rank, W), p + "mix.w2": (n, rank), p + "mix.w0": (n,),
                        p + "mix.u": (m["heads"], m["dim"]), p + "mix.norm": (n,), p + "mix.o": (W, n)})
        else:
            a, b = m["left"], m["right"]
            out.update({p + "mix.left.q": (a["heads"] * a["dim"], W), p + "mix.left.k": (a["kv_heads"] * a["dim"], W),
                        p + "mix.left.v": (a["kv_heads"] * a["vdim"], W), p + "mix.left.o": (W, a["heads"] * a["vdim"]),
                        p + "mix.right.q": (b["heads"] * b["dim"], W), p + "mix.right.k": (b["heads"] * b["dim"], W),
                        p + "mix.right.v": (b["heads"] * b["vdim"], W), p + "mix.right.g": (b["heads"] * b["vdim"], W),
                        p + "mix.right.o": (W, b["heads"] * b["vdim"]), p + "mix.right.norm": (b["heads"] * b["vdim"],)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(config, seed=0, rank=8):
    """Seeded bfloat16 weights under which every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config, rank).items():
        z = torch.randn(shape, generator=g)
        leaf = name.split(".", 1)[-1]
        if "norm" in leaf:
            z = 1 + 0.2 * z
        elif ".mu." in name:
            z = torch.rand(shape, generator=g)
        elif name.endswith(".w0"):
            z = -2 + 1.5 * z
        elif name.endswith(".u"):
            z = 0.5 * z
        elif name == "embed":
            z = z * 0.7
        else:
            z = z * shape[-1] ** -0.5
            if leaf in ("mix.left.q", "mix.left.k"):
                z = 1.5 * z
        out[name] = z.to(torch.bfloat16)
    return out


def widened(weights, dtype=torch.float64):
    return {k: v.to(dtype) for k, v in weights.items()}

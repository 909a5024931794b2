"""Plain, slow restatement of the Zuvulorn decoder in torch on the CPU.  TEST INFRASTRUCTURE ONLY.

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


def layer_norm(x, eps, weight):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(x, taps, bias=None):
    """x: (T, C), taps: (C, K).  Channel by channel; the last tap meets the current token, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            src = t - (K - 1 - j)
            if src >= 0:
                out[t] = out[t] + taps[:, j] * x[src]
    return out if bias is None else out + bias


def frequencies(dims, base, scaling=None):
    """Angular frequency per pair; with `scaling`, slow pairs are slowed by `factor` (three bands by wavelength)."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wavelength = 2 * math.pi / f
            if wavelength > original / low:
                f = f / factor
            elif wavelength >= original / high:
                s = (original / wavelength - low) / (high - low)
                f = (1 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate(x, position, dims, freqs):
    """x: (heads, dim) of one token; the first `dims` channels turn, pair (i, i + dims / 2)."""
    half = dims // 2
    angle = torch.tensor([position * f for f in freqs], dtype=torch.float64)
    c, s = torch.cos(angle).to(x.dtype), torch.sin(angle).to(x.dtype)
    u, v, rest = x[:, :half], x[:, half:dims], x[:, dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], 1)


def sink_attention(q, k, v, scale):
    """q: (T, H, d), k: (T, G, d), v: (T, G, e): causal; a score of 0 without a value stands beside the keys' scores."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        for h in range(H):
            g = h // (H // G)
            score = (k[:i + 1, g] @ q[i, h]) * scale
            top = max(score.max().item(), 0.0)
            e = torch.exp(score - top)
            out[i, h] = (e / (e.sum() + math.exp(-top))) @ v[:i + 1, g]
    return out


def rglru_gates(u, ra, ra_b, ri, ri_b, lam):
    """u: (T, C), ra / ri: (blocks, n, n).  (log of the decay, input gate), each (T, C)."""
    blocks, n, _ = ra.shape
    parts = u.view(u.shape[0], blocks, n)
    r = torch.sigmoid(torch.einsum("bij,tbj->tbi", ra, parts) + ra_b).reshape(u.shape)
    i = torch.sigmoid(torch.einsum("bij,tbj->tbi", ri, parts) + ri_b).reshape(u.shape)
    return -8 * r * softplus(lam), i


def gated_accumulation(log_a, drive):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) drive_t from S = 0; all states (T, C)."""
    state = torch.zeros_like(drive[0])
    out = []
    for t in range(drive.shape[0]):
        a = torch.exp(log_a[t])
        state = a * state + torch.sqrt(1 - a * a) * drive[t]
        out.append(state)
    return torch.stack(out)


def delta_memory(q, k, v, g, beta):
    """q, k, g: (T, H, d), v: (T, H, e), beta: (T, H).  Decay the rows, correct what k reads towards v, read with q."""
    T, H, d = q.shape
    state = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        state = g[t][:, :, None] * state
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", state, k[t]))
        state = state + torch.einsum("hd,he->hde", k[t], u)
        out.append(torch.einsum("hde,hd->he", state, q[t]))
    return torch.stack(out), state


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


# ------------------------------------------------------------------------------------------------
# mixers, feed-forward, model
# ------------------------------------------------------------------------------------------------
def rglru_mixer(w, pre, h, cfg, eps, kept):
    y = gelu_tanh(h @ w[pre + "y"].T + w[pre + "y.b"])
    u = short_conv(h @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    log_a, i = rglru_gates(u, w[pre + "ra"], w[pre + "ra.b"], w[pre + "ri"], w[pre + "ri.b"], w[pre + "lam"])
    return (gated_accumulation(log_a, i * u) * y) @ w[pre + "o"].T


def attention_mixer(w, pre, h, cfg, eps, kept):
    T = h.shape[0]
    H, G, d, e = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    rot = cfg["rot"]
    freqs = frequencies(rot["dims"], rot["base"], rot.get("scaling"))

    def turned(x):
        return torch.stack([rotate(x[t], t, rot["dims"], freqs) for t in range(T)])

    q = turned(rms_norm(h @ w[pre + "q"].T, eps, w[pre + "q.norm"]).view(T, H, d))
    if cfg.get("kv_from") is None:
        k = turned(rms_norm(h @ w[pre + "k"].T, eps, w[pre + "k.norm"]).view(T, G, d))
        v = (h @ w[pre + "v"].T).view(T, G, e)
        kept[pre] = k, v
    else:
        k, v = kept[f"l{cfg['kv_from']}.mix."]
    o = sink_attention(q, k, v, cfg["scale"]) * torch.sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * e) @ w[pre + "o"].T


def delta_mixer(w, pre, h, cfg, eps, kept):
    T = h.shape[0]
    H, G, d, e = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (silu(short_conv(h @ w[pre + s].T, w[pre + s + ".conv"])) for s in "qkv")
    q = unit(q.view(T, G, d)) * d ** -0.5
    k = unit(k.view(T, G, d))
    group = torch.arange(H) // (H // G)
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    rate = softplus((h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "dt_bias"]).view(T, H, d)
    g = torch.exp(-torch.exp(w[pre + "A_log"])[None, :, None] * rate)
    o, _ = delta_memory(q[:, group], k[:, group], v.view(T, H, e), g, beta)
    gate = torch.sigmoid((h @ w[pre + "g1"].T) @ w[pre + "g2"].T).view(T, H, e)
    o = rms_norm(o, eps, w[pre + "norm"]) * gate
    return o.reshape(T, H * e) @ w[pre + "o"].T


def experts_ff(w, pre, h, cfg):
    """Every token goes to the `top` experts with the largest sigmoid scores; the score scales the expert's input."""
    n, top = cfg["router"]["experts"], cfg["router"]["top"]
    score = torch.sigmoid(h @ w[pre + "router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in sorted(range(n), key=lambda e: -score[t, e].item())[:top]:
            z = score[t, e] * h[t]
            p = f"{pre}e{e}."
            out[t] = out[t] + w[p + "down"] @ (silu(w[p + "gate"] @ z) * (w[p + "up"] @ z))
    return out


MIXERS = {"rglru": rglru_mixer, "attention": attention_mixer, "channel_delta": delta_mixer}


def through(streams, w, pre, sublayer):
    """One sublayer between the streams (a list of (T, W)): mixed input, then all streams at once from the old ones."""
    n = len(streams)
    u = sum(w[pre + "in"][s] * streams[s] for s in range(n))
    y = sublayer(u)
    return [sum(w[pre + "mix"][s, t] * streams[s] for s in range(n)) + w[pre + "out"][t] * y for t in range(n)]


def forward(config, weights, tokens, keep_layers=False):
    """Logits (T, vocab) of one sequence; with keep_layers also the sum of the streams after every layer."""
    eps, w = config["norm"]["eps"], weights
    streams = [w["embed"][torch.as_tensor(tokens)]] * config["streams"]
    kept, memory = [], {}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        mixer = MIXERS[layer["type"]]
        streams = through(streams, w, p + "hc1.", lambda u: mixer(w, p + "mix.", layer_norm(u, eps, w[p + "norm1"]), layer["mixer"],
                                                                  eps, memory))
        if layer.get("mlp") is not None:
            streams = through(streams, w, p + "hc2.", lambda u: experts_ff(w, p + "mlp.", layer_norm(u, eps, w[p + "norm2"]), layer["mlp"]))
        kept.append(sum(streams))
    logits = layer_norm(sum(streams), eps, w["final.norm"]) @ w["head"].T
    return (logits, kept) if keep_layers else logits


# ------------------------------------------------------------------------------------------------
# small models for tests
# ------------------------------------------------------------------------------------------------
def tensor_shapes(config, rank=8):
    """name -> shape of every tensor a configuration needs; `rank` is the inner width of the low-rank paths."""
    W, V, S = config["width"], config["vocab"], config["streams"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        x = p + "mix."
        out[p + "norm1"] = (W,)
        if layer["type"] == "rglru":
            n, b = m["width"], m["blocks"]
            out.update({x + "y": (n, W), x + "y.b": (n,), x + "x": (n, W), x + "x.b": (n,), x + "conv": (n, m["conv"]), x + "conv.b": (n,),
                        x + "ra": (b, n // b, n // b), x + "ra.b": (b, n // b), x + "ri": (b, n // b, n // b), x + "ri.b": (b, n // b),
                        x + "lam": (n,), x + "o": (W, n)})
        elif layer["type"] == "attention":
            nq, nk, nv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            out.update({x + "q": (nq, W), x + "q.norm": (nq,), x + "g": (m["heads"], W), x + "o": (W, m["heads"] * m["vdim"])})
            if m.get("kv_from") is None:
                out.update({x + "k": (nk, W), x + "k.norm": (nk,), x + "v": (nv, W)})
        else:
            nk, nv, nd = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"] * m["dim"]
            for s, n in (("q", nk), ("k", nk), ("v", nv)):
                out.update({x + s: (n, W), x + s + ".conv": (n, m["conv"])})
            out.update({x + "b": (m["heads"], W), x + "A_log": (m["heads"],), x + "dt_bias": (nd,), x + "norm": (m["vdim"],),
                        x + "a1": (rank, W), x + "a2": (nd, rank), x + "g1": (rank, W), x + "g2": (nv, rank), x + "o": (W, nv)})
        subs = [1]
        if layer.get("mlp") is not None:
            ff, n = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]["experts"]
            subs.append(2)
            out.update({p + "norm2": (W,), p + "mlp.router": (n, W)})
            for e in range(n):
                out.update({f"{p}mlp.e{e}.gate": (ff, W), f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
        for q in subs:
            out.update({f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
    return out


def random_weights(config, seed=0, rank=8):
    """Seeded bfloat16 weights under which every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    S, out = config["streams"], {}
    for name, shape in tensor_shapes(config, rank).items():
        z = torch.randn(shape, generator=g)
        leaf = name.split(".", 1)[-1]
        if "norm" in leaf:
            z = 1 + 0.2 * z
        elif leaf in ("hc1.in", "hc2.in"):
            z = (1 + 0.4 * z) / S
        elif leaf in ("hc1.out", "hc2.out"):
            z = 1 + 0.4 * z
        elif leaf in ("hc1.mix", "hc2.mix"):
            z = 0.8 * torch.eye(S) + 0.2 / S + 0.1 * z
        elif leaf == "mix.lam":
            z = -2 + 1.5 * z
        elif leaf in ("mix.A_log", "mix.dt_bias"):
            z = -1 + z
        elif leaf.endswith(".b") and len(shape) < 2 or leaf in ("mix.ra.b", "mix.ri.b"):
            z = 0.5 * z
        elif leaf == "mlp.router":
            z = 3 * z * shape[-1] ** -0.5
        elif leaf != "embed":
            z = z * shape[-1] ** -0.5
        out[name] = z.to(torch.bfloat16)
    return out


def widened(weights, dtype=torch.float64):
    return {k: v.to(dtype) for k, v in weights.items()}

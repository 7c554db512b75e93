"""Plain, slow restatement of the Sigisun architecture for the tests: one function per mechanism, token by token where
the equations are, in the floating-point type of its inputs (float64 unless a test says otherwise). It shares no code
with ``openrlhf_b200``; weights are a dict of tensors keyed like a checkpoint, the configuration is the parsed
``config.json`` dict."""
import math

import torch


def rms_norm(x, weight, eps):
    """x [..., n]: divide by the root of (mean square + eps), then scale per channel."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def group_rms_norm(x, weight, groups, eps):
    """RMS norm in `groups` equal contiguous parts of the last axis, each with its own mean square."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * weight


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def causal_conv(u, weight, bias):
    """u [T, C], weight [C, taps]: out[t, c] = bias[c] + sum_k weight[c, k] u[t - (taps - 1) + k, c]; zeros before 0."""
    taps = weight.shape[1]
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        acc = bias.clone()
        for k in range(taps):
            s = t - (taps - 1) + k
            if s >= 0:
                acc = acc + weight[:, k] * u[s]
        out[t] = acc
    return out


def ssd_recurrence(x, b, c, dt, a_log, d, state=None):
    """x [T, heads, P], b / c [T, groups, N], dt [T, heads] (after softplus). Returns (y [T, heads, P], last state
    [heads, N, P]); the state starts at zero unless one is passed in."""
    T, H, P = x.shape
    G, N = b.shape[1], b.shape[2]
    s = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            decay = torch.exp(-torch.exp(a_log[h]) * dt[t, h])
            s[h] = decay * s[h] + dt[t, h] * torch.outer(b[t, g], x[t, h])
            y[t, h] = s[h].T @ c[t, g] + d[h] * x[t, h]
    return y, s


def mamba2_mixer(h, w, pre, m, eps):
    """h [T, width] (normalised input of the layer) -> mixer output [T, width]."""
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = h @ w[pre + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    assert dt.shape[1] == H
    xbc = silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x = xbc[:, :inner].reshape(-1, H, P)
    b = xbc[:, inner:inner + G * N].reshape(-1, G, N)
    c = xbc[:, inner + G * N:].reshape(-1, G, N)
    dt = softplus(dt + w[pre + "dt_bias"])
    y, _ = ssd_recurrence(x, b, c, dt, w[pre + "A_log"], w[pre + "D"])
    y = y.reshape(-1, inner) * silu(z)
    return group_rms_norm(y, w[pre + "norm"], m["norm_groups"], eps) @ w[pre + "o"].T


def rotary(x, positions, dims, base, factor):
    """x [T, heads, D]: rotate (i, i + dims/2) of the first `dims` channels by position * base^(-2i/dims) / factor."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = positions.to(x.dtype) * (base ** (-2.0 * i / dims) / factor)
        cos, sin = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * cos - v * sin
        out[:, :, i + half] = v * cos + u * sin
    return out


def visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def sink_softmax(scores):
    """Weights over the last axis with an extra valueless entry of score 0 in the denominator."""
    m = scores.max(-1, keepdim=True).values.clamp_min(0)
    e = torch.exp(scores - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def windowed_attention(q, k, v, scale, size, keep_first):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(i + 1) if visible(i, j, size, keep_first)]
        for h in range(H):
            g = h // rep
            p = sink_softmax((k[js, g] @ q[i, h]) * scale)
            out[i, h] = p @ v[js, g]
    return out


def attention_mixer(h, w, pre, m, shared_kv):
    """Returns (mixer output, (rotated keys, values)); `shared_kv` replaces the layer's own keys and values."""
    T = h.shape[0]
    pos = torch.arange(T)
    rot = m["rot"]
    turn = lambda t: rotary(t, pos, rot["dims"], rot["base"], rot["scaling"]["factor"])
    q = turn((h @ w[pre + "q"].T).reshape(T, m["heads"], m["dim"]))
    if shared_kv is None:
        k = turn((h @ w[pre + "k"].T).reshape(T, m["kv_heads"], m["dim"]))
        v = (h @ w[pre + "v"].T).reshape(T, m["kv_heads"], m["vdim"])
    else:
        k, v = shared_kv
    a = windowed_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["keep_first"])
    return a.reshape(T, -1) @ w[pre + "o"].T, (k, v)


def relu2_mlp(h, w, pre):
    return torch.relu(h @ w[pre + "up"].T) ** 2 @ w[pre + "down"].T


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer, [layers, T, width])."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kv, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        h = rms_norm(x, w[f"l{i}.norm1"], eps)
        pre, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "mamba2":
            y = mamba2_mixer(h, w, pre, m, eps)
        else:
            src = m.get("kv_from")
            y, kv[i] = attention_mixer(h, w, pre, m, None if src is None else kv[src])
        if layer.get("mlp") is not None:
            y = y + relu2_mlp(h, w, f"l{i}.mlp.")
        x = x + y
        after.append(x)
    logits = softcap(rms_norm(x, w["final.norm"], eps) @ w["head"].T, cfg["logit_softcap"])
    return (logits, torch.stack(after)) if want_layers else logits


def random_weights(cfg, seed=0):
    """bf16-representable random weights in a checkpoint's layout."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, k=None: (torch.randn(*s, generator=g) / math.sqrt(s[-1] if k is None else k)).to(torch.bfloat16)
    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": r(V, W, k=1), "head": r(V, W) * 3, "final.norm": 1 + 0.2 * r(W, k=1)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        w[p + "norm1"] = 1 + 0.2 * r(W, k=1)
        if layer["type"] == "mamba2":
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            w[p + "mix.in"] = r(2 * inner + 2 * gn + m["heads"], W)
            w[p + "mix.conv"] = r(inner + 2 * gn, m["conv"])
            w[p + "mix.conv.b"] = 0.1 * r(inner + 2 * gn, k=1)
            w[p + "mix.dt_bias"] = (torch.rand(m["heads"], generator=g) * 4 - 4).to(torch.bfloat16)
            w[p + "mix.A_log"] = (torch.rand(m["heads"], generator=g) * 2.5 - 1).to(torch.bfloat16)
            w[p + "mix.D"] = r(m["heads"], k=1)
            w[p + "mix.norm"] = 1 + 0.2 * r(inner, k=1)
            w[p + "mix.o"] = r(W, inner)
        else:
            w[p + "mix.q"] = 2 * r(m["heads"] * m["dim"], W)
            if m.get("kv_from") is None:
                w[p + "mix.k"] = 2 * r(m["kv_heads"] * m["dim"], W)
                w[p + "mix.v"] = r(m["kv_heads"] * m["vdim"], W)
            w[p + "mix.o"] = r(W, m["heads"] * m["vdim"])
        if layer.get("mlp") is not None:
            w[p + "mlp.up"] = r(layer["mlp"]["ff"], W)
            w[p + "mlp.down"] = r(W, layer["mlp"]["ff"])
    return {k: v.to(torch.bfloat16) for k, v in w.items()}

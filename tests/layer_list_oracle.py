"""Plain implementation of the layer-list models (windowed attention with a whole-projection q/k norm, Mamba-2,
gated dense feed-forward, post-sublayer norms), one function per mechanism, written from the equations.

It works on a whole sequence at once, keeps no cache, loops over tokens where the mechanism is a recurrence, and takes
its weights by their checkpoint names from a plain dictionary.  Nothing of the package is imported.  Everything is
computed in the dtype of ``DT`` (double by default)."""
import math

import torch

DT = torch.float64


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def rotate(x, positions, dims, base, factor=1.0):
    """Rotate-half rotation of the first ``dims`` entries of every head; x [T, heads, dim]."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        f = base ** (-2.0 * i / dims) / factor
        a = positions.to(DT) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def softmax_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] of one sequence -> [T, H, dv]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    hide = j > i
    if window is not None:
        hide = hide | (i - j >= window)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(hide, -math.inf)
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (p / p.sum(-1, keepdim=True)) @ v[:, g]
    return out


def project_keys_values(h, w, p, m, eps):
    """Keys (normed over the whole projection, rotated) and values of a layer with its own projections."""
    T = h.shape[0]
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).view(T, m["kv_heads"], m["dim"])
    v = (h @ w[p + "v"].T).view(T, m["kv_heads"], m["vdim"])
    return rope_of(k, m), v


def rope_of(x, m):
    rot = m.get("rot")
    if not rot:
        return x
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    return rotate(x, torch.arange(x.shape[0]), rot["dims"], rot["base"], factor)


def attention_mixer(h, w, p, m, eps, kv):
    """``kv``: the (keys, values) this layer attends to, its own or another layer's."""
    T = h.shape[0]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, m["heads"], m["dim"])
    q = rope_of(q, m)
    window = (m.get("mask") or {}).get("size")
    o = softmax_attention(q, kv[0], kv[1], m["scale"], window)
    return o.reshape(T, -1) @ w[p + "o"].T


def causal_conv(x, weight, bias):
    """Per-channel causal convolution, x [T, C], weight [C, taps] (last column = current token)."""
    T, taps = x.shape[0], weight.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = bias.clone()
        for k in range(taps):
            s = t - (taps - 1 - k)
            if s >= 0:
                acc = acc + weight[:, k] * x[s]
        out[t] = acc
    return out


def ssm_scan(x, B, C, dt, A_log, D, state=None):
    """The recurrence: x [T, H, P], B / C [T, G, N], dt [T, H] (after softplus) -> y [T, H, P], final S [H, N, P]."""
    T, H, P = x.shape
    G, N = B.shape[1], B.shape[2]
    S = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.zeros_like(x)
    of = torch.arange(H) // (H // G)
    decay = torch.exp(-torch.exp(A_log)[None, :] * dt)
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][of][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t][of][:, :, None]).sum(1) + D[:, None] * x[t]
    return y, S


def gated_group_norm(y, z, w, parts, eps):
    """(y * silu(z)) normed in ``parts`` equal pieces, each by its own root mean square, times w."""
    g = y * silu(z)
    T, n = g.shape
    gp = g.view(T, parts, n // parts)
    gp = gp / torch.sqrt((gp * gp).mean(-1, keepdim=True) + eps)
    return gp.reshape(T, n) * w


def mamba2_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:inner + inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].view(T, H, P)
    B = xbc[:, inner:inner + G * N].view(T, G, N)
    C = xbc[:, inner + G * N:].view(T, G, N)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=1e9)
    y, _ = ssm_scan(x, B, C, dt, w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


def feed_forward(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, weights, tokens, trace=None):
    """Logits [T, vocab] of one token sequence.  ``trace``: list that receives the residual after every layer."""
    w = {k: v.to(DT) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    kvs = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        if L["type"].startswith("attention"):
            src = m.get("kv_from")
            if src is None:
                kvs[i] = project_keys_values(x, w, p, m, eps)
            y = attention_mixer(x, w, p, m, eps, kvs[i if src is None else src])
        else:
            y = mamba2_mixer(x, w, p, m, eps)
        x = x + rms_norm(y, w[f"l{i}.norm1"], eps)
        if L.get("mlp"):
            x = x + rms_norm(feed_forward(x, w, f"l{i}.mlp."), w[f"l{i}.norm2"], eps)
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]

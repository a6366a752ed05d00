"""Plain implementation of the Fimudra design: layer norms ahead of the sublayers, several residual streams with learned
mixing, WKV time mixing, softmax attention with a sink beside a matrix memory (mLSTM), and a mixture of clamped gated experts
with identity experts and a shared one.  One function per mechanism, written from the equations.

Whole sequences at once, no cache, loops over tokens where the mechanism is a recurrence, weights by their checkpoint names
from a plain dictionary.  Nothing of the package is imported.  Computed in ``DT``."""
import math

import torch

DT = torch.float64


def layer_norm(x, w, eps):
    """Centred and scaled to unit variance (population), times w."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def log_sigmoid(z):
    return torch.where(z < 0, z, torch.zeros_like(z)) - torch.log1p(torch.exp(-z.abs()))


# ----------------------------------------------------------------------------- residual streams
def gather_streams(x, weights):
    """x [T, s, W] -> [T, W], the sublayer's input before its norm."""
    return sum(weights[s] * x[:, s] for s in range(x.shape[1]))


def spread_streams(x, mix, out, y):
    """Every stream anew from all old ones (``mix[from, to]``) and the sublayer's output."""
    new = torch.empty_like(x)
    for t in range(x.shape[1]):
        new[:, t] = out[t] * y
        for s in range(x.shape[1]):
            new[:, t] = new[:, t] + mix[s, t] * x[:, s]
    return new


# ----------------------------------------------------------------------------- attention with a sink
def frequency(i, dims, base, scaling):
    f = base ** (-2.0 * i / dims)
    if not scaling:
        return f
    length = 2 * math.pi / f
    orig, low, high, factor = (float(scaling[k]) for k in ("original", "low", "high", "factor"))
    if length < orig / high:
        return f
    if length > orig / low:
        return f / factor
    s = (orig / length - low) / (high - low)
    return (1 - s) * f / factor + s * f


def rotate(x, positions, rot):
    """Rotate-half on the first ``dims`` entries of every head; x [T, heads, dim]."""
    if not rot:
        return x
    half, out = rot["dims"] // 2, x.clone()
    for i in range(half):
        a = positions.to(x.dtype) * frequency(i, rot["dims"], rot["base"], rot.get("scaling"))
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i], out[:, :, i + half] = u * c - v * s, v * c + u * s
    return out


def sink_attention(q, k, v, scale, sink):
    """Causal; exp(sink) of the head stands in every softmax sum without a key or a value."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    hide = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    for h in range(H):
        s = ((q[:, h] @ k[:, h // per].T) * scale).masked_fill(hide, -math.inf)
        top = torch.maximum(s.max(-1).values, sink[h])[:, None]
        e = torch.exp(s - top)
        out[:, h] = (e / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - top))) @ v[:, h // per]
    return out


def attention_mixer(h, w, p, m):
    T = h.shape[0]
    pos = torch.arange(T)
    q = rotate((h @ w[p + "q"].T).view(T, m["heads"], m["dim"]), pos, m.get("rot"))
    k = rotate((h @ w[p + "k"].T).view(T, m["kv_heads"], m["dim"]), pos, m.get("rot"))
    v = (h @ w[p + "v"].T).view(T, m["kv_heads"], m["vdim"])
    return sink_attention(q, k, v, m["scale"], w[p + "sink"]).reshape(T, -1) @ w[p + "o"].T


# ----------------------------------------------------------------------------- matrix memory
def capped(z, cap):
    return cap * torch.tanh(z / cap)


def matrix_memory(q, k, v, log_in, log_forget):
    """q, k [T, H, N], v [T, H, P], gates [T, H] -> o [T, H, P]."""
    T, H, N = q.shape
    S, n, m = torch.zeros(H, N, v.shape[2], dtype=q.dtype), torch.zeros(H, N, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        new = torch.maximum(log_forget[t] + m, log_in[t])
        keep, add = torch.exp(log_forget[t] + m - new)[:, None], torch.exp(log_in[t] - new)[:, None]
        S = keep[:, :, None] * S + add[:, :, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep * n + add * k[t]
        m = new
        top = torch.einsum("hnp,hn->hp", S, q[t])
        out[t] = top / (torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6)[:, None]
    return out


def mlstm_mixer(h, w, p, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, N) / math.sqrt(N)
    k, v = (h @ w[p + "k"].T).view(T, H, N), (h @ w[p + "v"].T).view(T, H, P)
    i = capped(h @ w[p + "i"].T + w[p + "i.b"], m["gate_cap"])
    f = log_sigmoid(capped(h @ w[p + "f"].T + w[p + "f.b"], m["gate_cap"]))
    o = unit_rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * P)
    return (o * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    return (m["left_scale"] * attention_mixer(h, w, p + "left.", m["left"])
            + m["right_scale"] * mlstm_mixer(h, w, p + "right.", m["right"], eps))


# ----------------------------------------------------------------------------- WKV
def token_shift(h):
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv_scan(r, k, v, decay, u, S=None):
    """r, k, decay [T, H, N], v [T, H, P], u [H, N] -> o [T, H, P], final S."""
    T, H, N = r.shape
    S = torch.zeros(H, N, v.shape[2], dtype=r.dtype) if S is None else S
    out = torch.zeros_like(v)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hnp,hn->hp", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return out, S


def wkv_mixer(h, w, p, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    prev = token_shift(h)
    mixed = {c: h + (prev - h) * w[p + "mu." + c] for c in "rkvgw"}
    r, k, v = ((mixed[c] @ w[p + c].T).view(T, H, D) for c in "rkv")
    gate = mixed["g"] @ w[p + "g"].T
    gate = gate * sigmoid(gate)
    decay = torch.exp(-torch.exp(torch.tanh(mixed["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(T, H, D)
    o, _ = wkv_scan(r, k, v, decay, w[p + "u"])
    return (unit_rms(o, eps).reshape(T, H * D) * w[p + "norm"] * gate) @ w[p + "o"].T


# ----------------------------------------------------------------------------- feed-forward
def clamped_glu(h, w, p, limit):
    g = torch.minimum(h @ w[p + "gate"].T, torch.tensor(limit, dtype=h.dtype))
    u = (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def choose(z, correction, top, scale):
    """Router logits [T, E] -> per token {expert: weight}."""
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    picks = []
    for t in range(z.shape[0]):
        order = sorted(range(z.shape[1]), key=lambda j: -float(s[t, j] + correction[j]))
        picks.append({j: float(s[t, j]) * scale for j in order[:top]})
    return picks


def expert_mixture(h, w, p, m):
    r, E = m["router"], m["router"]["experts"]
    out = torch.zeros_like(h)
    for t, pick in enumerate(choose(h @ w[p + "router"].T, w[p + "correction"], r["top"], r["scale"])):
        for j, weight in pick.items():
            out[t] += weight * (clamped_glu(h[t:t + 1], w, f"{p}e{j}.", m["expert"]["limit"])[0] if j < E else h[t])
    if m.get("shared"):
        out = out + clamped_glu(h, w, p + "shared.", m["shared"]["limit"])
    return out


# ----------------------------------------------------------------------------- the model
MIXERS = {"parallel": parallel_mixer, "wkv": wkv_mixer}


def forward(cfg, weights, tokens, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace``: list that receives the sum of the streams after every layer."""
    w = {k: v.to(DT) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = (w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"])[:, None].repeat(1, cfg["streams"], 1)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{L.get('weights_of', i)}."
        subs = [(1, lambda h: MIXERS[L["type"].split("_")[0]](h, w, p + "mix.", L["mixer"], eps))]
        if L.get("mlp"):
            subs.append((2, lambda h: expert_mixture(h, w, p + "mlp.", L["mlp"])))
        for q, sub in subs:
            hc = f"{p}hc{q}."
            y = sub(layer_norm(gather_streams(x, w[hc + "in"]), w[f"{p}norm{q}"], eps))
            x = spread_streams(x, w[hc + "mix"], w[hc + "out"], y)
        if trace is not None:
            trace.append(x.sum(1))
    return layer_norm(x.sum(1), w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]

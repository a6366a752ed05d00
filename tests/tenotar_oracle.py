"""Plain implementation of the Tenotar design: one residual with norms ahead of the sublayers; attention through a query and a
key/value latent with an output gate; windowed attention with kept first tokens, per-head norms and pairwise rotation; chunked
attention with convolved projections, capped scores and a distance bias; values mixed with those of an earlier layer; gated
feed-forwards, dense or a mixture with a shared expert.  One function per mechanism, written from the equations.

Whole sequences at once, no cache, weights by their checkpoint names from a plain dictionary.  Nothing of the package is
imported.  Computed in ``DT``."""
import math

import torch

DT = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def linear(h, w, name):
    """With the bias of that name, if there is one."""
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


# ----------------------------------------------------------------------------- positions
def rotate(x, rot, pairs):
    """x [T, heads, dim], rows at positions 0, 1, ...; ``pairs``: (i, j) of every rotated pair, in order of frequency."""
    out, pos = x.clone(), torch.arange(x.shape[0], dtype=x.dtype)
    for n, (i, j) in enumerate(pairs):
        a = pos * rot["base"] ** (-2.0 * n / rot["dims"])
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        out[:, :, i], out[:, :, j] = x[:, :, i] * c - x[:, :, j] * s, x[:, :, j] * c + x[:, :, i] * s
    return out


def halves(dims):
    return [(i, i + dims // 2) for i in range(dims // 2)]


def neighbours(dims):
    return [(2 * i, 2 * i + 1) for i in range(dims // 2)]


# ----------------------------------------------------------------------------- which keys a query sees
def _grid(T):
    return torch.arange(T)[:, None], torch.arange(T)[None, :]


def window_mask(T, size, keep_first=0):
    i, j = _grid(T)
    return (j <= i) & ((i - j < size) | (j < keep_first))


def chunk_mask(T, size):
    i, j = _grid(T)
    return (j <= i) & (i // size == j // size)


# ----------------------------------------------------------------------------- softmax attention
def attend(q, k, v, scale, see, softcap=None, slopes=None):
    """q [T, H, D], k [T, G, D], v [T, G, P], ``see`` [T, T] -> [T, H, P]."""
    T, H, _ = q.shape
    per, out = H // k.shape[1], []
    i, j = _grid(T)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        if slopes is not None:
            s = s - slopes[h] * (i - j)
        out.append(torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, h // per])
    return torch.stack(out, 1)


def slopes_of(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def short_conv(u, taps):
    """y_t = sum_j taps[:, j] u_{t - n + 1 + j}, zeros ahead of the sequence."""
    n = taps.shape[1]
    pad = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=u.dtype), u])
    return sum(taps[:, j] * pad[j:j + u.shape[0]] for j in range(n))


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


# ----------------------------------------------------------------------------- mixers: (h, w, prefix, sizes, eps, first values)
def latent_mixer(h, w, p, m, eps, shared):
    T, H, D, R, P = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = ((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :m["kv_rank"]], eps) * w[p + "dkv.norm"]
    qr = rotate(q[:, :, D:], m["rot"], halves(R))
    kr = rotate(down[:, None, m["kv_rank"]:], m["rot"], halves(R))
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, D), kr.expand(T, H, R)], -1)
    o = attend(torch.cat([q[:, :, :D], qr], -1), k, (c @ w[p + "uv"].T).view(T, H, P), m["scale"], window_mask(T, m["mask"]["size"]))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * P) @ w[p + "o"].T


def _mixed(v, w, p, m, shared):
    if not m.get("v_mix"):
        return v
    if "first" not in shared:
        shared["first"] = v
        return v
    return mix_values(v, shared["first"], w[p + "vmix"])


def window_mixer(h, w, p, m, eps, shared):
    T, H, G, D, P = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(linear(h, w, p + "q").view(T, H, D), eps) * w[p + "q.norm"]
    k = rms(linear(h, w, p + "k").view(T, G, D), eps) * w[p + "k.norm"]
    v = _mixed(linear(h, w, p + "v"), w, p, m, shared).view(T, G, P)
    pairs = neighbours(m["rot"]["dims"])
    o = attend(rotate(q, m["rot"], pairs), rotate(k, m["rot"], pairs), v, m["scale"],
               window_mask(T, m["mask"]["size"], m["mask"].get("keep_first", 0)))
    return linear(o.reshape(T, H * P), w, p + "o")


def chunk_mixer(h, w, p, m, eps, shared):
    T, H, G, D, P = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ w[p + c].T, w[p + c + ".conv"]) for c in "qkv")
    v = _mixed(v, w, p, m, shared)
    o = attend(q.view(T, H, D), k.view(T, G, D), v.view(T, G, P), m["scale"], chunk_mask(T, m["mask"]["size"]), m["softcap"], slopes_of(H))
    return o.reshape(T, H * P) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_mixer, "attention": window_mixer, "attention_2": chunk_mixer}


# ----------------------------------------------------------------------------- feed-forward
def gated(h, w, p):
    return linear(silu(linear(h, w, p + "gate")) * linear(h, w, p + "up"), w, p + "down")


def choose(z, top):
    """Logits [T, E] -> per token {expert: weight}, the softmax over the chosen logits."""
    picks = []
    for row in z:
        best = sorted(range(len(row)), key=lambda e: -float(row[e]))[:top]
        picks.append(dict(zip(best, torch.softmax(row[best], 0).tolist())))
    return picks


def mixture(h, w, p, m):
    out = torch.zeros_like(h)
    for t, pick in enumerate(choose(linear(h, w, p + "router"), m["router"]["top"])):
        for e, weight in pick.items():
            out[t] += weight * gated(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out + gated(h, w, p + "shared.") if m.get("shared") else out


# ----------------------------------------------------------------------------- the model
def forward(cfg, weights, tokens, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace``: list that receives the residual after every layer."""
    w = {k: v.to(DT) for k, v in weights.items()}
    eps, shared = cfg["norm"]["eps"], {}
    x = w["embed"][torch.as_tensor(tokens)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[L["type"]](rms(x, eps) * w[p + "norm1"], w, p + "mix.", L["mixer"], eps, shared)
        if L.get("mlp"):
            h = rms(x, eps) * w[p + "norm2"]
            x = x + (mixture if L["mlp"]["kind"] == "moe" else lambda h, w, p, m: gated(h, w, p))(h, w, p + "mlp.", L["mlp"])
        if trace is not None:
            trace.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T * cfg.get("logit_scale", 1.0)


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]

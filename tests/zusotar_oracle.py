"""Plain implementation of the Zusotar design: one residual with norms ahead of and behind every sublayer and a learned average over
depth after every layer; attention over a key/value latent with a sink; windowed attention with normed values, a logarithmic
distance bias and an output gate; gated linear attention; gated feed-forwards, dense or a group-limited sigmoid mixture with a shared
expert; learned positions.  One function per mechanism, written from the equations.

Whole sequences at once, no cache, weights by their checkpoint names from a plain dictionary.  Nothing of the package is
imported.  Computed in ``DT``."""
import torch

DT = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    return rms(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ----------------------------------------------------------------------------- embedding, connection of the layers
def embed(tokens, w):
    t = torch.as_tensor(tokens)
    return w["embed"][t] + w["pos"][:len(t)]


def depth_average(weights, results):
    """``results``: the embedding output and what every layer so far gave."""
    return sum(weights[j] * r for j, r in enumerate(results))


# ----------------------------------------------------------------------------- rotation
def rotate_neighbours(x, dims, base):
    """x [T, heads, dim], rows at positions 0, 1, ...; entries 2i and 2i + 1 of the first ``dims`` turn together."""
    out, pos = x.clone(), torch.arange(x.shape[0], dtype=x.dtype)
    for i in range(dims // 2):
        a = (pos * base ** (-2.0 * i / dims))[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return out


# ----------------------------------------------------------------------------- which keys a query sees, and its softmax
def _distance(T):
    return torch.arange(T)[:, None] - torch.arange(T)[None, :]


def causal_mask(T):
    return _distance(T) >= 0


def window_mask(T, size):
    return (_distance(T) >= 0) & (_distance(T) < size)


def distance_bias(T, r1, r2):
    """[heads, T, T], taken off the scores (of visible keys)."""
    d = _distance(T).clamp_min(0).to(r1.dtype)
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * d)


def softmax_values(scores, mask, v, sink=None):
    """scores [heads, T, T], v [T, heads, vdim] -> [T, heads, vdim]."""
    s = scores.masked_fill(~mask, float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(-1, s.shape[1], 1)], -1)
    p = torch.softmax(s, -1)[..., :v.shape[0]]
    return torch.einsum("hij,jhv->ihv", p, v)


# ----------------------------------------------------------------------------- mixers
def latent_attention(h, w, p, m, eps):
    T, H, d, r, c = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    kv = h @ w[p + "dkv"].T
    lat = rms(kv[:, :c], eps) * w[p + "dkv.norm"]
    base = m["rot"]["base"]
    kr = rotate_neighbours(kv[:, None, c:], r, base)[:, 0]
    qr = rotate_neighbours(q[:, :, d:], r, base)
    k = (lat @ w[p + "uk"].T).view(T, H, d)
    v = (lat @ w[p + "uv"].T).view(T, H, m["vdim"])
    s = (torch.einsum("ihd,jhd->hij", q[:, :, :d], k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    return softmax_values(s, causal_mask(T), v, w[p + "sink"]).reshape(T, -1) @ w[p + "o"].T


def attention(h, w, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).view(T, H, m["dim"])
    k = (h @ w[p + "k"].T).view(T, G, m["dim"]).repeat_interleave(H // G, 1)
    v = rms((h @ w[p + "v"].T).view(T, G, m["vdim"]), eps).repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] - distance_bias(T, w[p + "r1"], w[p + "r2"])
    o = softmax_values(s, window_mask(T, m["mask"]["size"]), v).reshape(T, -1)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def gla_scan(q, k, v, alpha, S=None):
    """q, k, alpha [T, H, N], v [T, H, P] -> (o [T, H, P], state [H, N, P])."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if S is None else S
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, q[t]))
    return torch.stack(out), S


def gla_decay(z, tau):
    return sigmoid(z) ** (1.0 / tau)


def gla(h, w, p, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (h @ w[p + "q"].T).view(T, H, N) * N ** -0.5, (h @ w[p + "k"].T).view(T, H, N)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    o, _ = gla_scan(q, k, (h @ w[p + "v"].T).view(T, H, P), gla_decay(z, m["tau"]).view(T, H, N))
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * P)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "attention": attention, "gla": gla}


# ----------------------------------------------------------------------------- feed-forwards
def gated_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, router):
    """Router logits [T, experts] -> (chosen [T, top], weights [T, top])."""
    s = sigmoid(z)
    pick = s.clone()
    g = router.get("groups")
    if g:
        by_group = s.view(s.shape[0], g["count"], -1)
        score = by_group.topk(min(2, by_group.shape[2]), -1).values.sum(-1)
        for t in range(s.shape[0]):
            best = set(score[t].topk(g["keep"]).indices.tolist())
            for e in range(s.shape[1]):
                if e // by_group.shape[2] not in best:
                    pick[t, e] = -1.0
    ids = pick.topk(router["top"], -1).indices
    return ids, s.gather(1, ids)


def mixture(h, w, p, mlp):
    ids, weights = route(h @ w[p + "router"].T, mlp["router"])
    out = gated_ff(h, w, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), weights[t]):
            out[t] = out[t] + a * gated_ff(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


# ----------------------------------------------------------------------------- the model
def forward(cfg, weights, tokens, with_layers=False):
    """``cfg``: the dictionary of a config.json, ``weights``: {name: tensor} -> logits [T, vocab]."""
    w = {k: v.to(DT) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embed(tokens, w)
    results, after = [x], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = MIXERS[layer["type"].rstrip("_0123456789")]
        x = x + m * norm_around_zero(mixer(norm_around_zero(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps),
                                     w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp:
            h = norm_around_zero(x, w[p + "norm2"], eps)
            y = mixture(h, w, p + "mlp.", mlp) if mlp.get("kind") == "moe" else gated_ff(h, w, p + "mlp.")
            x = x + m * norm_around_zero(y, w[p + "norm2b"], eps)
        results.append(x)
        x = depth_average(w[p + "dwa"], results)
        after.append(x)
    logits = norm_around_zero(x, w["final.norm"], eps) @ w["head"].T
    return (logits, after) if with_layers else logits

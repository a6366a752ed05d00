"""Small random layer-list models for the tests: configurations, weights under their checkpoint names, model folders."""
import json
import math

import torch

import layer_list_oracle as oracle


def attention(heads=4, kv_heads=2, dim=24, vdim=16, window=20, rot=8, base=10000.0, factor=2.0, kv_from=None, ff=40):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.3 / math.sqrt(dim)}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if factor != 1.0:
            m["rot"]["scaling"] = {"factor": factor}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def mamba(heads=4, vdim=16, state=24, groups=2, conv=4, norm_groups=2, ff=0, kind="mamba2"):
    m = {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}
    return {"type": kind, "mixer": m, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def config(layers, width=48, vocab=97, eps=1e-5):
    return {"architecture": "Forovik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# name -> configuration.  "plain" is the common shape; "odd" has sizes that are no multiple of 8, another order, a layer
# without window or rotation, one tap, one group, and feed-forwards where the others have none; "wide" takes the
# tensor-core paths of every kernel.
CONFIGS = {
    "plain": config([attention(), mamba(), mamba(heads=6, vdim=8, state=16, groups=3, kind="mamba2_2"),
                     attention(window=33, kv_from=0), mamba(norm_groups=1)]),
    "odd": config([mamba(heads=3, vdim=10, state=7, groups=1, conv=3, norm_groups=3, ff=21), attention(heads=3, kv_heads=1, dim=9,
                   vdim=5, window=7, rot=6, ff=0), mamba(heads=2, vdim=5, state=33, groups=2, conv=1, norm_groups=1),
                   attention(heads=5, kv_heads=5, dim=7, vdim=12, window=0, rot=0, ff=13),
                   attention(heads=3, kv_heads=1, dim=9, vdim=5, window=18, rot=6, kv_from=1, ff=30)], width=37, vocab=61, eps=1e-3),
    "wide": config([mamba(heads=4, vdim=40, state=72, groups=2, conv=2, norm_groups=4, ff=128),
                    attention(heads=8, kv_heads=2, dim=72, vdim=104, window=70, rot=72, base=5000.0, factor=1.0, ff=256),
                    attention(heads=8, kv_heads=2, dim=72, vdim=104, window=130, rot=72, base=5000.0, factor=1.0, kv_from=1, ff=0),
                    mamba(heads=2, vdim=64, state=160, groups=1, norm_groups=2)], width=136, vocab=203),
}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}
    mat = lambda o, i, s=1.0: torch.randn(o, i, generator=g) * (s / math.sqrt(i))        # noqa: E731
    norm = lambda n: 1 + 0.2 * torch.randn(n, generator=g)                                # noqa: E731
    w["embed"] = torch.randn(cfg["vocab"], W, generator=g) * 0.6
    w["final.norm"] = norm(W) * 0.7
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        w[p + "norm1"] = norm(W) * 0.6
        if L["type"].startswith("attention"):
            q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            w[p + "mix.q"], w[p + "mix.q.norm"] = mat(q, W), norm(q) * 1.5
            w[p + "mix.o"] = mat(W, m["heads"] * m["vdim"])
            if m.get("kv_from") is None:
                w[p + "mix.k"], w[p + "mix.v"], w[p + "mix.k.norm"] = mat(k, W), mat(v, W), norm(k) * 1.5
        else:
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            C = inner + 2 * gn
            w[p + "mix.in"] = mat(inner + C + m["heads"], W)
            w[p + "mix.conv"] = torch.randn(C, m["conv"], generator=g) * 0.5
            w[p + "mix.conv.b"] = torch.randn(C, generator=g) * 0.1
            w[p + "mix.dt_bias"] = torch.randn(m["heads"], generator=g) * 0.5 - 1.5
            w[p + "mix.A_log"] = torch.randn(m["heads"], generator=g) * 0.7 - 0.5
            w[p + "mix.D"] = torch.randn(m["heads"], generator=g)
            w[p + "mix.norm"] = norm(inner)
            w[p + "mix.o"] = mat(W, inner)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            w[p + "norm2"] = norm(W) * 0.6
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(ff, W, 1.5), mat(ff, W), mat(W, ff)
    return {k: v.to(dtype) for k, v in w.items()}


def write_model(folder, cfg, w):
    from safetensors.torch import save_file
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(folder / "model.safetensors"))


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(got, want):
    """Per row: difference (mean taken off, root mean square) over the spread of the expected logits."""
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def error(got, want):
    """Largest row error; for a bf16 run a row may be several times off the typical one from rounding alone."""
    return float(row_errors(got, want).max())


_cache: dict = {}


def expected(name, seed, toks):
    """Oracle logits of every position (remembered: several tests ask for the same sequences)."""
    key = (name, seed, tuple(toks))
    if key not in _cache:
        _cache[key] = oracle.forward(CONFIGS[name], weights(CONFIGS[name], seed), toks)
    return _cache[key]

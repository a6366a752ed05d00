"""Small random models of the Fimudra design for the tests: configurations, and weights under their checkpoint names."""
import math

import torch

import fimudra_oracle as oracle


def moe(experts=5, identity=2, top=3, ff=24, limit=1.5, shared=40, shared_limit=0.8, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared, "limit": shared_limit} if shared else None,
            "router": {"experts": experts, "identity": identity, "scale": scale, "top": top}}


def parallel(heads=4, kv_heads=2, dim=24, vdim=16, rot=8, base=500.0, scaling=(4.0, 1.0, 4.0, 128), m_heads=3, m_dim=16, m_vdim=24, cap=9.0,
             left_scale=0.7, right_scale=1.3, mlp="moe", kind="parallel"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.3 / math.sqrt(dim)}
    if rot:
        left["rot"] = {"dims": rot, "base": base}
        if scaling:
            left["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    m = {"left": left, "left_scale": left_scale, "right_scale": right_scale,
         "right": {"heads": m_heads, "dim": m_dim, "vdim": m_vdim, "gate_cap": cap}}
    return {"type": kind, "mixer": m, "mlp": moe() if mlp == "moe" else mlp}


def wkv(heads=3, dim=16, mlp="moe", kind="wkv"):
    return {"type": kind, "mixer": {"heads": heads, "dim": dim}, "mlp": moe() if mlp == "moe" else mlp}


def config(layers, width=48, vocab=97, eps=1e-5, streams=2, scale=5.0):
    return {"architecture": "Fimudra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams,
            "embedding": {"scale": scale}}


def all_of(**kw):
    """Every expert is chosen: rounding cannot move a choice."""
    return moe(experts=4, identity=2, top=6, **kw)


# "plain": the common shape, every kind of layer and one that runs with an earlier layer's weights.  "odd": sizes that are no
# multiple of 8, three streams, a layer without feed-forward, a mixture without shared and one without identity experts, another
# order, weights taken from a later layer, rotation of all and of no dimensions.  "wide": the tensor-core paths of every kernel.
CONFIGS = {
    "plain": config([parallel(mlp=all_of()), wkv(mlp=all_of()), parallel(m_heads=2, m_dim=24, mlp=moe(), kind="parallel_2"), wkv(heads=2, dim=24),
                     dict(parallel(mlp=all_of()), weights_of=0)]),
    "odd": config([dict(wkv(heads=2, dim=9, mlp=moe(3, 1, 2, 13, 0.9, 0)), weights_of=2),
                   parallel(heads=3, kv_heads=1, dim=9, vdim=5, rot=0, m_heads=2, m_dim=7, m_vdim=11, cap=3.0, mlp=None),
                   wkv(heads=2, dim=9, mlp=moe(3, 1, 2, 13, 0.9, 0)),
                   parallel(heads=5, kv_heads=5, dim=6, vdim=12, rot=6, scaling=None, m_heads=1, m_dim=33, m_vdim=5, left_scale=1.0,
                            right_scale=0.4, mlp=moe(6, 0, 1, 21, 2.0, 17, 3.0, 0.6))], width=37, vocab=61, eps=1e-3, streams=3, scale=0.7),
    "wide": config([wkv(heads=2, dim=64, mlp=all_of(ff=128, shared=128)),
                    parallel(heads=8, kv_heads=2, dim=72, vdim=104, rot=72, base=5000.0, m_heads=2, m_dim=64, m_vdim=128, mlp=all_of(ff=64, shared=256)),
                    dict(wkv(heads=2, dim=64, mlp=all_of(ff=128, shared=128)), weights_of=0),
                    parallel(heads=4, kv_heads=4, dim=64, vdim=64, m_heads=3, m_dim=128, m_vdim=72, mlp=None),
                    wkv(heads=1, dim=128, mlp=None)], width=136, vocab=203, streams=4, scale=2.0),
}
RANK = 6      # of the decay's projection: only the tensors tell


def weights(cfg, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    W, n, w = cfg["width"], cfg["streams"], {}
    mat = lambda o, i, s=1.0: torch.randn(o, i, generator=g) * (s / math.sqrt(i))        # noqa: E731
    vec = lambda k, s=1.0, m=0.0: m + s * torch.randn(k, generator=g)                    # noqa: E731
    w["embed"] = torch.randn(cfg["vocab"], W, generator=g) * 0.6
    w["final.norm"] = vec(W, 0.2, 1)
    for i, L in enumerate(cfg["layers"]):
        if "weights_of" in L:
            continue
        p, m = f"l{i}.", L["mixer"]
        for q in (1, 2) if L["mlp"] else (1,):
            w[p + f"norm{q}"] = vec(W, 0.2, 1)
            w[p + f"hc{q}.in"], w[p + f"hc{q}.out"] = vec(n, 0.3, 0.6), vec(n, 0.3, 0.8)
            w[p + f"hc{q}.mix"] = 0.9 * torch.eye(n) + 0.15 * torch.randn(n, n, generator=g)
        if L["type"].startswith("parallel"):
            a, r, lp, rp = m["left"], m["right"], p + "mix.left.", p + "mix.right."
            w[lp + "q"], w[lp + "k"] = mat(a["heads"] * a["dim"], W, 1.5), mat(a["kv_heads"] * a["dim"], W, 1.5)
            w[lp + "v"], w[lp + "o"] = mat(a["kv_heads"] * a["vdim"], W), mat(W, a["heads"] * a["vdim"])
            w[lp + "sink"] = vec(a["heads"], 2.0, 1.0)
            k, v = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            w[rp + "q"], w[rp + "k"], w[rp + "v"], w[rp + "g"] = mat(k, W), mat(k, W), mat(v, W), mat(v, W)
            w[rp + "o"], w[rp + "norm"] = mat(W, v), vec(v, 0.2, 1)
            w[rp + "i"], w[rp + "f"] = mat(r["heads"], W, 2.0), mat(r["heads"], W)
            w[rp + "i.b"], w[rp + "f.b"] = vec(r["heads"], 1.0, -1.0), vec(r["heads"], 1.0, 3.0)
        else:
            k = m["heads"] * m["dim"]
            for c in "rkvgw":
                w[p + "mix.mu." + c] = torch.rand(W, generator=g)
            for c in "rkvg":
                w[p + "mix." + c] = mat(k, W)
            w[p + "mix.w1"], w[p + "mix.w2"], w[p + "mix.w0"] = mat(RANK, W), mat(k, RANK, 0.7), vec(k, 1.5, -2.5)
            w[p + "mix.u"], w[p + "mix.norm"], w[p + "mix.o"] = torch.randn(m["heads"], m["dim"], generator=g), vec(k, 0.2, 1), mat(W, k)
        if L["mlp"]:
            f, r = L["mlp"], L["mlp"]["router"]
            w[p + "mlp.router"], w[p + "mlp.correction"] = mat(r["experts"] + r["identity"], W, 1.5), vec(r["experts"] + r["identity"], 0.2)
            names = [(f"e{e}", f["expert"]["ff"]) for e in range(r["experts"])] + ([("shared", f["shared"]["ff"])] if f["shared"] else [])
            for e, ff in names:
                q = f"{p}mlp.{e}."
                w[q + "gate"], w[q + "up"], w[q + "down"] = mat(ff, W, 2.0), mat(ff, W, 1.5), mat(W, ff)
    return {k: v.to(dtype) for k, v in w.items()}


_cache: dict = {}


def expected(name, seed, toks):
    key = (name, seed, tuple(toks))
    if key not in _cache:
        _cache[key] = oracle.forward(CONFIGS[name], weights(CONFIGS[name], seed), toks)
    return _cache[key]

"""Small random models of the Zusotar design for the tests: configurations, and weights under their checkpoint names."""
import math

import torch

import zusotar_oracle as oracle


def moe(experts=6, top=2, ff=24, shared=40, groups=(3, 2)):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None, "router": router}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def all_of(**kw):
    """Every expert is chosen: rounding cannot move a choice."""
    return moe(experts=4, top=4, groups=(2, 2), **kw)


def latent(heads=3, dim=16, rot=8, vdim=24, kv_rank=32, base=300.0, mlp="moe", name="latent_attention"):
    return {"type": name, "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot},
                      "scale": 1.2 / math.sqrt(dim + rot)}}


def window(heads=4, kv_heads=2, dim=24, vdim=16, size=20, mlp="moe", name="attention"):
    return {"type": name, "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": 0.9 / math.sqrt(dim)}}


def gla(heads=3, dim=16, vdim=24, tau=5.0, rank=12, mlp="moe", name="gla"):
    return {"type": name, "mlp": moe() if mlp == "moe" else mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "_rank": rank}


def config(layers, width=48, vocab=97, eps=1e-5, mult=0.6, positions=512):
    return {"architecture": "Zusotar", "layers": [{k: v for k, v in L.items() if k != "_rank"} for L in layers], "norm": {"eps": eps},
            "vocab": vocab, "width": width, "residual_mult": mult, "max_positions": positions, "_ranks": [L.get("_rank") for L in layers]}


# "plain": every kind of layer, one of them twice with other sizes.  "odd": sizes that are no multiple of 8, windows of one, one key
# channel, layers without feed-forward, shared expert or groups, another order.  "wide": the tensor-core paths of every kernel, several
# chunks of the head sizes, windows over pages, many value columns.  "deep": latents of the size that the latent decode kernel is made
# for, and a smaller one stored so; the largest key size of the chunked recurrence.
CONFIGS = {
    "plain": config([latent(mlp=dense()), gla(), window(), latent(heads=2, dim=24, vdim=8, kv_rank=48, base=900.0, mlp=all_of(), name="latent_attention_2"),
                     window(heads=2, kv_heads=2, dim=16, size=9, name="attention_2"), gla(heads=2, dim=24, vdim=16, tau=16.0, rank=8, mlp=dense(32))]),
    "odd": config([gla(heads=5, dim=7, vdim=13, tau=1.0, rank=5, mlp=moe(3, 3, 13, 0, None)),
                   window(heads=3, kv_heads=1, dim=9, vdim=15, size=1, mlp=None),
                   latent(heads=5, dim=7, rot=6, vdim=5, kv_rank=13, base=50.0, mlp=moe(6, 6, 21, 17, (2, 2))),
                   window(heads=3, kv_heads=3, dim=11, vdim=5, size=64, mlp=dense(21)),
                   gla(heads=1, dim=3, vdim=9, tau=0.4, rank=1, mlp=None),
                   latent(heads=1, dim=3, rot=2, vdim=13, kv_rank=3, mlp=moe(2, 2, 8, 3, (1, 1)))],
                  width=37, vocab=61, eps=1e-3, mult=0.8, positions=301),
    "wide": config([window(heads=8, kv_heads=2, dim=72, vdim=104, size=70, mlp=dense(128)),
                    latent(heads=4, dim=128, rot=64, vdim=128, kv_rank=192, mlp=all_of(ff=128, shared=256)),
                    gla(heads=2, dim=64, vdim=136, tau=16.0, rank=16, mlp=None),
                    window(heads=16, kv_heads=2, dim=136, vdim=64, size=129, mlp=None),
                    gla(heads=3, dim=40, vdim=64, tau=2.0, rank=24, mlp=all_of(ff=64, shared=0)),
                    latent(heads=20, dim=64, rot=32, vdim=72, kv_rank=96, mlp=None)], width=136, vocab=203, mult=0.3),
    "deep": config([latent(heads=6, dim=32, rot=64, vdim=40, kv_rank=512, mlp=dense(48)),
                    gla(heads=1, dim=256, vdim=40, tau=8.0, mlp=None),
                    latent(heads=3, dim=24, rot=16, vdim=32, kv_rank=260, mlp=None)], width=64, vocab=80),
}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}
    mat = lambda o, i, s=1.0: torch.randn(o, i, generator=g) * (s / math.sqrt(i))        # noqa: E731
    vec = lambda k, s=1.0, m=0.0: m + s * torch.randn(k, generator=g)                    # noqa: E731
    w["embed"], w["pos"] = torch.randn(cfg["vocab"], W, generator=g) * 0.6, torch.randn(cfg["max_positions"], W, generator=g) * 0.3
    w["head"], w["final.norm"] = mat(cfg["vocab"], W, 2.0), vec(W, 0.2)
    for i, L in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", L["mixer"], L["type"].rstrip("_0123456789")
        x, H = p + "mix.", m["heads"]
        w[p + "norm1"], w[p + "norm1b"] = vec(W, 0.2), vec(W, 0.2)
        w[p + "dwa"] = vec(i + 2, 0.3)
        w[p + "dwa"][-1] += 1.0
        if kind == "latent_attention":
            w[x + "q"], w[x + "dkv"] = mat(H * (m["dim"] + m["rot_dim"]), W, 1.5), mat(m["kv_rank"] + m["rot_dim"], W, 1.2)
            w[x + "dkv.norm"], w[x + "sink"] = vec(m["kv_rank"], 0.2, 1), vec(H, 1.5)
            w[x + "uk"], w[x + "uv"] = mat(H * m["dim"], m["kv_rank"], 1.5), mat(H * m["vdim"], m["kv_rank"])
        elif kind == "attention":
            w[x + "q"], w[x + "k"] = mat(H * m["dim"], W, 1.3), mat(m["kv_heads"] * m["dim"], W, 1.3)
            w[x + "v"], w[x + "g"] = mat(m["kv_heads"] * m["vdim"], W, 0.02), mat(H * m["vdim"], W, 1.5)       # eps of their norm counts
            w[x + "r1"], w[x + "r2"] = vec(H, 0.5, 0.6), torch.exp(vec(H, 1.0, -1.0))
        else:
            n, v, rank = H * m["dim"], H * m["vdim"], cfg["_ranks"][i]
            w[x + "q"], w[x + "k"], w[x + "v"], w[x + "g"] = mat(n, W, 1.5), mat(n, W, 1.2), mat(v, W), mat(v, W, 1.5)
            w[x + "a1"], w[x + "a2"], w[x + "a2.b"], w[x + "norm"] = mat(rank, W), mat(n, rank, 1.5), vec(n, 1.5, 1.0), vec(m["vdim"], 0.3, 1)
        w[x + "o"] = mat(W, H * m["vdim"])
        if L["mlp"]:
            f = L["mlp"]
            w[p + "norm2"], w[p + "norm2b"] = vec(W, 0.2), vec(W, 0.2)
            if f["kind"] == "dense":
                names = [("", f["ff"])]
            else:
                E = f["router"]["experts"]
                w[p + "mlp.router"] = mat(E, W, 1.5)
                names = [(f"e{e}.", f["expert"]["ff"]) for e in range(E)] + ([("shared.", f["shared"]["ff"])] if f["shared"] else [])
            for e, ff in names:
                q = f"{p}mlp.{e}"
                w[q + "gate"], w[q + "up"], w[q + "down"] = mat(ff, W, 1.5), mat(ff, W, 1.2), mat(W, ff)
    return {k: v.to(dtype) for k, v in w.items()}


_cache: dict = {}


def expected(name, seed, toks):
    key = (name, seed, tuple(toks))
    if key not in _cache:
        _cache[key] = oracle.forward(CONFIGS[name], weights(CONFIGS[name], seed), toks)
    return _cache[key]

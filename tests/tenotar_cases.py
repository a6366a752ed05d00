"""Small random models of the Tenotar design for the tests: configurations, and weights under their checkpoint names."""
import math

import torch

import tenotar_oracle as oracle


def moe(experts=5, top=2, ff=24, shared=40):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None, "router": {"experts": experts, "top": top}}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def all_of(**kw):
    """Every expert is chosen: rounding cannot move a choice."""
    return moe(experts=4, top=4, **kw)


def latent(heads=3, dim=16, rot=8, vdim=24, q_rank=40, kv_rank=32, window=20, base=300.0, mlp="moe"):
    return {"type": "latent_attention", "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot}, "scale": 1.2 / math.sqrt(dim + rot)}}


def window(heads=4, kv_heads=2, dim=24, vdim=16, size=20, keep=3, rot=16, base=700.0, v_mix=True, mlp="moe"):
    return {"type": "attention", "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep},
                      "rot": {"base": base, "dims": rot}, "scale": 0.9 / math.sqrt(dim), "v_mix": v_mix}}


def chunk(heads=4, kv_heads=2, dim=16, vdim=16, size=30, conv=3, cap=4.0, v_mix=True, mlp="moe"):
    return {"type": "attention_2", "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "conv": conv, "softcap": cap,
                      "scale": 1.4 / math.sqrt(dim), "v_mix": v_mix}}


def config(layers, width=48, vocab=97, eps=1e-5, logit_scale=0.6):
    return {"architecture": "Tenotar", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": logit_scale}


# "plain": every kind of layer, the mixing of values handed on from one kind to the other.  "odd": sizes that are no multiple of
# 8, windows and chunks of one and of odd sizes, one tap, no kept tokens, layers without feed-forward or shared expert or mixing,
# another order, the first value layer a chunked one.  "wide": the tensor-core paths of every kernel, several chunks of the head
# sizes, windows over pages.  "deep": latents of the size that the latent decode kernel is made for, and a smaller one stored so.
CONFIGS = {
    "plain": config([latent(mlp=dense()), window(), chunk(), latent(window=33, mlp=all_of()), window(heads=2, kv_heads=2, dim=16, rot=16, keep=5, size=9),
                     chunk(conv=4, size=17, mlp=dense(32))]),
    "odd": config([chunk(heads=3, kv_heads=1, dim=9, vdim=15, size=7, conv=1, cap=1.5, mlp=moe(3, 3, 13, 0)),
                   latent(heads=5, dim=7, rot=6, vdim=5, q_rank=11, kv_rank=13, window=1, base=50.0, mlp=None),
                   window(heads=3, kv_heads=3, dim=11, vdim=5, size=5, keep=0, rot=6, mlp=dense(21)),
                   window(heads=3, kv_heads=1, dim=10, vdim=7, size=1, keep=9, rot=10, v_mix=False, mlp=moe(7, 7, 21, 17)),
                   chunk(heads=5, kv_heads=5, dim=6, vdim=3, size=40, conv=6, cap=30.0, mlp=None),
                   latent(heads=1, dim=3, rot=2, vdim=13, q_rank=5, kv_rank=3, window=64, mlp=moe(2, 2, 8, 3))],
                  width=37, vocab=61, eps=1e-3, logit_scale=2.5),
    "wide": config([window(heads=8, kv_heads=2, dim=72, vdim=104, size=70, keep=66, rot=40, mlp=dense(128)),
                    latent(heads=4, dim=128, rot=64, vdim=128, q_rank=96, kv_rank=192, window=100, mlp=all_of(ff=128, shared=256)),
                    chunk(heads=8, kv_heads=2, dim=136, vdim=104, size=129, conv=4, cap=15.0, mlp=None),
                    latent(heads=20, dim=64, rot=32, vdim=72, q_rank=64, kv_rank=96, window=65, mlp=all_of(ff=64, shared=0)),
                    chunk(heads=16, kv_heads=2, dim=64, vdim=104, size=64, conv=2, mlp=None)], width=136, vocab=203, logit_scale=1.0),
    "deep": config([latent(heads=6, dim=32, rot=64, vdim=40, q_rank=56, kv_rank=512, window=80, mlp=dense(48)),
                    latent(heads=3, dim=24, rot=16, vdim=32, q_rank=24, kv_rank=260, window=130, mlp=None)], width=64, vocab=80),
}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}
    mat = lambda o, i, s=1.0: torch.randn(o, i, generator=g) * (s / math.sqrt(i))        # noqa: E731
    vec = lambda k, s=1.0, m=0.0: m + s * torch.randn(k, generator=g)                    # noqa: E731
    w["embed"], w["head"], w["final.norm"] = torch.randn(cfg["vocab"], W, generator=g) * 0.6, mat(cfg["vocab"], W, 2.0), vec(W, 0.2, 1)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x, H = p + "mix.", m["heads"]
        w[p + "norm1"] = vec(W, 0.2, 1)
        if L["type"] == "latent_attention":
            w[x + "dq"], w[x + "dkv"], w[x + "g"] = mat(m["q_rank"], W), mat(m["kv_rank"] + m["rot_dim"], W), mat(H, W)
            w[x + "dq.norm"], w[x + "dkv.norm"] = vec(m["q_rank"], 0.2, 1), vec(m["kv_rank"], 0.2, 1)
            w[x + "uq"] = mat(H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
            w[x + "uk"], w[x + "uv"] = mat(H * m["dim"], m["kv_rank"], 1.5), mat(H * m["vdim"], m["kv_rank"])
        else:
            sizes = {"q": H * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for c, n in sizes.items():
                w[x + c] = mat(n, W, 1.3)
                if L["type"] == "attention":
                    w[x + c + ".b"] = vec(n, 0.3)
                else:
                    w[x + c + ".conv"] = vec((n, m["conv"]), 0.6)
            if L["type"] == "attention":
                w[x + "q.norm"], w[x + "k.norm"], w[x + "o.b"] = vec(m["dim"], 0.3, 1.5), vec(m["dim"], 0.3, 1.5), vec(W, 0.2)
            if m["v_mix"]:
                w[x + "vmix"] = 0.2 + 0.6 * torch.rand((), generator=g)
        w[x + "o"] = mat(W, H * m["vdim"])
        if L["mlp"]:
            f = L["mlp"]
            w[p + "norm2"] = vec(W, 0.2, 1)
            if f["kind"] == "dense":
                names = [("", f["ff"])]
                w[p + "mlp.gate.b"], w[p + "mlp.up.b"], w[p + "mlp.down.b"] = vec(f["ff"], 0.4), vec(f["ff"], 0.4), vec(W, 0.3)
            else:
                E = f["router"]["experts"]
                w[p + "mlp.router"], w[p + "mlp.router.b"] = mat(E, W, 1.5), vec(E, 0.5)
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

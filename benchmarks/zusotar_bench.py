#!/usr/bin/env python
"""The Zusotar design (latent attention with sinks, gated linear attention, windowed attention with a logarithmic bias, expert mixtures,
norms on both sides of the sublayers, averages over depth) beside the framework's closest models at equal sizes, random weights.

    python bench.py --layer-list zusotar-kernels    each kernel against its roofline, beside the like kernel of the other models
    python bench.py --layer-list zusotar-model      prefill and decode throughput through the engine, beside an MLA and a GQA expert model
    python bench.py --layer-list zusotar            both

Timing as in ``layer_list_bench.py``."""
from __future__ import annotations

import json

from .layer_list_bench import PEAKS, Timer
from .tenotar_bench import CASES, mla_like, qwen_like, throughput

SIZES = {
    "2k": dict(width=2048, layers=12, heads=16, kv_heads=4, dim=128, kv_rank=512, rot_dim=64, window=1024, g_heads=16, g_dim=64, g_vdim=128, g_rank=16,
               ff=5632, experts=32, groups=4, keep=2, top=4, expert_ff=768, shared_ff=1536, vocab=32768),
    "4k": dict(width=4096, layers=6, heads=32, kv_heads=8, dim=128, kv_rank=512, rot_dim=64, window=1024, g_heads=16, g_dim=128, g_vdim=256, g_rank=16,
               ff=11264, experts=64, groups=8, keep=4, top=6, expert_ff=1024, shared_ff=2048, vocab=32768),
}


def kernels(out) -> None:
    import torch

    from omni_infer_b200 import ops
    from omni_infer_b200.ops import _native as nat
    from omni_infer_b200.ops import attention as A
    from omni_infer_b200.ops import attn_prepare as ap
    from omni_infer_b200.ops import depth
    from omni_infer_b200.ops import layer_list as ll
    from omni_infer_b200.ops import matrix_state as ms
    from omni_infer_b200.ops import streams as st
    timer, dev = Timer(), "cuda"
    torch.manual_seed(0)
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.5).bfloat16()        # noqa: E731
    f32 = lambda *s: torch.randn(*s, device=dev)                          # noqa: E731

    def row(size, what, name, fn, nbytes, flops=0.0):
        us = timer(fn)
        nat.check_status()
        t = max(nbytes / (PEAKS["hbm_gbs"] * 1e3), flops / (PEAKS["bf16_tflops"] * 1e6))
        out({"size": size, "case": what, "kernel": name, "us": round(us, 1), "GB/s": round(nbytes / us / 1e3),
             "TFLOP/s": round(flops / us / 1e6, 1), "roofline": round(t / us, 3)})

    for size, c in SIZES.items():
        W, H, G, D, win, n_l = c["width"], c["heads"], c["kv_heads"], c["dim"], c["window"], c["layers"]
        C, R, eps = c["kv_rank"], c["rot_dim"], 1e-5
        for what, B, L in CASES:
            pre = what.startswith("prefill")
            T = B * L if pre else B
            bs, nblk = 128, (L + 127) // 128
            bt = torch.arange(1, B * nblk + 1, dtype=torch.int32, device=dev).view(B, nblk)
            pos = (torch.arange(L, device=dev).repeat(B) if pre else torch.full((B,), L - 1, device=dev)).contiguous()
            seq = torch.arange(B, dtype=torch.int32, device=dev).repeat_interleave(T // B)
            slots = bt[seq.long(), pos // bs].long() * bs + pos % bs
            cu = torch.arange(B + 1, dtype=torch.int32, device=dev) * (T // B)
            sl = torch.full((B,), L, dtype=torch.int32, device=dev)
            ss = torch.arange(B, dtype=torch.int32, device=dev)
            cq = cu if pre else None
            seen_w = min(win, L)
            pairs_w = B * (seen_w * (seen_w + 1) / 2 + (L - seen_w) * seen_w) if pre else B * seen_w
            pairs = B * L * (L + 1) / 2 if pre else B * L
            # ---- embedding, norms on both sides, averages
            ids, emb, posn = torch.randint(0, c["vocab"], (T,), device=dev), bf(c["vocab"], W), bf(8192, W)
            x, y, one, yr, wb = f32(T, W), bf(T, W), torch.ones(W, device=dev), bf(T, W), torch.ones(W, device=dev).bfloat16()
            row(size, what, "embed_positions", lambda: depth.embed_positions(ids, emb, pos, posn, x, one, eps, ld=W), T * W * 10)
            row(size, what, "  like: embed_norm", lambda: ll.embed_norm(ids, emb, one, eps, ld=W), T * W * 8)
            step = lambda y_, **k: depth.both_norms_step(x, x, y_, one, 0.4, one, eps, torch.bfloat16, ld=W, **k)      # noqa: E731
            row(size, what, "both_norms_step (within a layer)", lambda: step(y), T * W * 12)
            res = f32(n_l, T, W)
            for n in (1, n_l // 2, n_l):
                avg = torch.full((n + 1,), 1.0 / (n + 1), device=dev)
                row(size, what, f"both_norms_step (average of {n + 1})", lambda: step(y, results=res, average=avg), T * W * (12 + 4 * n + 4 * (n < n_l)))
            row(size, what, "  like: post_norm_add", lambda: ll.post_norm_add(y, one, x, eps), T * W * 12)
            row(size, what, "  like: rmsnorm + residual", lambda: ops.rmsnorm(y, wb, eps, residual=yr), T * W * 8)
            del res, emb, posn
            # ---- windowed attention
            h0, nq = bf(T, W), (2 * H + 2 * G) * D      # with the gate's columns
            wq = bf(nq, W)
            row(size, what, "q, k, v, gate gemm (the same kernel)", lambda: ops.gemm(h0, wq), (nq * W + T * W + T * nq) * 2, 2.0 * T * W * nq)
            del wq
            kc, vc, qkv = bf(B * nblk + 1, bs, G, D), bf(B * nblk + 1, bs, G, D), bf(T, nq)
            cs = ops.rope_cos_sin_table(D, 8200, 5e5, None, device=dev)
            qnb = torch.ones(D, device=dev).bfloat16()
            row(size, what, "qkv_prepare (cache write, normed values)",
                lambda: ap.qkv_prepare(qkv, H, G, D, D, None, None, eps, None, 0, False, pos, slots, kc, vc, v_norm=True), T * 4 * G * D * 2)
            q0 = qkv[:, : (H + 2 * G) * D].contiguous()
            row(size, what, "  like: rope_qk_cache (per-head norm)", lambda: ops.rope_qk_cache(q0, H, G, D, cs, pos, slots, kc, vc, qnb, qnb, eps),
                T * ((H + G) * 2 + 2 * G) * D * 2)
            del q0
            q3, gate = qkv[:, : H * D].unflatten(1, (H, D)), qkv[:, (H + 2 * G) * D:]
            bias = (torch.full((H,), 0.5, device=dev), torch.linspace(0.01, 1.0, H, device=dev))
            kw = dict(positions=pos, q_to_seq=seq, slots=slots, block_table=bt, seq_lens=sl, scale=D ** -0.5, cu_q=cq, max_q=T // B, max_seq_len=L)
            io = lambda seen, g=1: T * ((2 + g) * H + 2 * G) * D * 2 if pre else (B * seen * 2 * G + (2 + g) * B * H) * D * 2      # noqa: E731
            row(size, what, f"attention, window {win}, log bias, gated", lambda: ll.paged_attention(q3, kc, vc, window=win, log_bias=bias, gate=gate, **kw),
                io(seen_w), pairs_w * H * 4 * D)
            row(size, what, "attention, log bias, gated (all keys)", lambda: ll.paged_attention(q3, kc, vc, log_bias=bias, gate=gate, **kw), io(L),
                pairs * H * 4 * D)
            if pre:
                k3, v3 = qkv[:, H * D:(H + G) * D].unflatten(1, (G, D)), qkv[:, (H + G) * D:(H + 2 * G) * D].unflatten(1, (G, D))
                row(size, what, "  like: gqa_prefill", lambda: A.gqa_prefill(q3, k3, v3, cu, cu, D ** -0.5, L, L), io(L, 0), pairs * H * 4 * D)
            else:
                qc = q3.contiguous()
                row(size, what, "  like: gqa_decode", lambda: A.gqa_decode(qc, kc, vc, bt, sl, D ** -0.5, L), io(L, 0), pairs * H * 4 * D)
            del kc, vc, qkv, q3, gate
            # ---- latent attention
            n = H * (D + R)
            a, cache = bf(T, n + C + R), bf(B * nblk + 1, bs, C + R)
            csr = ops.rope_cos_sin_table(R, 8200, 1e4, None, device=dev)
            cw, sink = torch.ones(C, device=dev), f32(H)
            cwb = cw.bfloat16()
            row(size, what, "latent_prepare", lambda: ap.latent_prepare(a, 0, n, C, R, None, cw, eps, csr, pos, slots, cache, C, 0, pre),
                T * (C + R) * (2 + pre) * 2)
            q = a[:, :n].unflatten(1, (H, D + R))
            row(size, what, "rotate_heads", lambda: ap.rotate_heads(q[..., D:], R, csr, pos, q[..., D:]), T * H * R * 4)
            qd = bf(T, H, D + R)
            row(size, what, "  like: mla_kv_rope_cache (with the queries' rotation)",
                lambda: ops.mla_kv_rope_cache(a[:, n:], cwb, eps, csr, pos, slots, cache, q=qd, q_rope_off=D, want_latent=pre),
                T * ((C + R) * (2 + pre) + 2 * H * R) * 2)
            if pre:
                rows_, wkv = bf(T, C + R), bf(H * 2 * D, C)
                kv = ops.gemm(rows_[:, :C], wkv)
                s0, s1 = cu[:-1], cu[1:]
                seg = dict(d1=D, dv=D, q_start=s0, q_end=s1, k_start=s0, k_end=s1, max_q=L, scale=(D + R) ** -0.5)
                by, fl = T * (H * (D + R + 2 * D + D) + R) * 2, H * 2.0 * (D + R + D)
                row(size, what, "latent_prefill, sinks", lambda: ap.latent_prefill(q, kv, rows_[:, C:], sink=sink, **seg), by, pairs * fl)
                row(size, what, "  like: mla_prefill", lambda: A.mla_prefill(qd, kv, rows_, H, D, R, D, cu, cu, (D + R) ** -0.5, L, L), by, pairs * fl)
                del rows_, wkv, kv
            else:
                qa = bf(T, H, C + R)
                lat = dict(positions=pos, q_to_seq=seq, slots=slots, block_table=bt, seq_lens=sl, scale=(D + R) ** -0.5, max_seq_len=L)
                by, fl = (B * L * (C + R) + T * H * (2 * C + R)) * 2, H * 2.0 * (2 * C + R)
                row(size, what, "latent_attention, sinks", lambda: ap.latent_attention(qa, cache, C, sink=sink, **lat), by, B * L * fl)
                row(size, what, "  like: mla_decode", lambda: ops.mla_decode(qa, cache, bt, sl, (D + R) ** -0.5, max_seq_len=L), by, B * L * fl)
                del qa
            del a, cache, q, qd
            # ---- gated linear attention, beside WKV with heads of its key size and as many values in all
            GH, N, P = c["g_heads"], c["g_dim"], c["g_vdim"]
            p1 = pos if pre else torch.full_like(pos, L)
            rec, span = dict(positions=p1, state_slots=ss, cu_q=cq), dict(min_q=T // B, max_q=T // B)
            nk, nv = GH * N, GH * P
            a2, ua, zb = bf(nk, c["g_rank"]), bf(T, 64), f32(nk)
            row(size, what, "decay gemm", lambda: ops.gemm(ua[:, :c["g_rank"]], a2, out_dtype=torch.float32), T * (c["g_rank"] * 2 + nk * 4))
            qk, v, z, S = bf(T, 2 * nk), bf(T, nv), f32(T, nk), torch.zeros(B, GH, P, N, device=dev)
            by, fl = T * (2 * nk + 2 * nv) * 2 + T * nk * 4 + S.numel() * 4 * (1 if pre else 2), T * GH * 64 * 2.0 * (N + P) / 2 + T * GH * 4.0 * N * P
            row(size, what, "gla_scan", lambda: ms.gla_scan(qk[:, :nk], qk[:, nk:], v, z, zb, 1 / 16, S, H=GH, P=P, N=N, **rec, **span), by, fl if pre else 0)
            WH = nv // N
            r4, z4, w0, u4, S4 = bf(T, 3, nv), f32(T, nv), f32(nv), f32(nv), torch.zeros(B, WH, N, N, device=dev)
            by, fl = T * nv * 12 + S4.numel() * 4 * (1 if pre else 2), T * WH * (64 * 2.0 * N + 4.0 * N * N)
            row(size, what, "  like: wkv_scan", lambda: ms.wkv_scan(r4[:, 0], r4[:, 1], r4[:, 2], z4, w0, u4, S4, H=WH, N=N, **rec, **span), by,
                fl if pre else 0)
            yy, nw, oo = bf(T, nv), torch.ones(nv, device=dev), bf(T, nv)
            row(size, what, "head_norm (the same kernel)", lambda: ms.head_norm(yy, v, nw, oo, H=GH, P=P, eps=eps, act="silu"), T * nv * 6)
            del qk, v, z, S, r4, z4, S4, yy, oo
            # ---- experts
            E, k, ff = c["experts"], c["top"], c["expert_ff"]
            wr = bf(E, W) * 0.1
            lg = ops.gemm(h0, wr, out_dtype=torch.float32)
            how = dict(mode="sigmoid", n_group=c["groups"], topk_group=c["keep"], group_mode="top2sum")
            row(size, what, "router_topk (groups, sigmoid; the same kernel)", lambda: ops.router_topk(lg, k, **how), T * (E + 2 * k) * 4)
            ids_, wt = ops.router_topk(lg, k, **how)
            pm = ops.moe_permute(h0, ids_, wt, 0, E)
            n_rows = int(pm.seg_len.sum())
            w13, w2 = bf(E, 2 * ff, W), bf(E, W, ff)
            seg = dict(seg_start=pm.seg_start, seg_len=pm.seg_len, t_hint=max(16, (T * k + E - 1) // E))
            ye = ops.gemm(ops.gemm(pm.x, w13, epi="swiglu", **seg), w2, row_scale=pm.row_w, **seg)
            es = st.ExpertSum(ye, pm.row_of, ids_, wt, E, h0, y)
            res, avg = f32(n_l, T, W), torch.full((3,), 0.3, device=dev)
            row(size, what, "both_norms_step + expert sum (average of 3)", lambda: step(es, results=res, average=avg), T * W * 24 + n_rows * W * 2)
            row(size, what, "  like: moe_combine", lambda: ops.moe_combine(ye, pm.row_of, T, k, shared=y), T * W * 4 + n_rows * W * 2)
            del w13, w2, x, ye, pm, res, h0, y, es
            torch.cuda.empty_cache()


def models(out) -> None:
    from omni_infer_b200.models.config import zusotar
    for size, c in SIZES.items():
        for name, mc in (("zusotar", zusotar(**c)), ("mla-moe", mla_like(c)), ("qwen3-moe", qwen_like(c))):
            throughput(out, size, c, name, mc)


def main(which: str) -> int:
    def out(d):
        print(json.dumps(d), flush=True)
    if which in ("zusotar-kernels", "zusotar"):
        kernels(out)
    if which in ("zusotar-model", "zusotar"):
        models(out)
    return 0

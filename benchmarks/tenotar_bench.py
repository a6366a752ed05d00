#!/usr/bin/env python
"""The Tenotar design (latent, windowed and chunked attention, expert mixtures, norms ahead of the sublayers) beside the framework's
closest models at equal sizes, random weights.

    python bench.py --layer-list tenotar-kernels    each kernel against its roofline, beside the like kernel of the other models
    python bench.py --layer-list tenotar-model      prefill and decode throughput through the engine, beside an MLA and a GQA expert model
    python bench.py --layer-list tenotar            both

Timing as in ``layer_list_bench.py``."""
from __future__ import annotations

import json

from .layer_list_bench import PEAKS, Timer

SIZES = {
    "2k": dict(width=2048, layers=12, heads=16, kv_heads=4, dim=128, q_rank=768, kv_rank=512, rot_dim=64, window=1024, keep_first=4,
               chunk=1024, conv=4, ff=5632, experts=32, top=4, expert_ff=768, shared_ff=1536, vocab=32768),
    "4k": dict(width=4096, layers=6, heads=32, kv_heads=8, dim=128, q_rank=1536, kv_rank=512, rot_dim=64, window=1024, keep_first=4,
               chunk=1024, conv=4, ff=11264, experts=64, top=6, expert_ff=1024, shared_ff=2048, vocab=32768),
}
CASES = (("prefill 8x1024", 8, 1024), ("prefill 1x8192", 1, 8192), ("decode 64 @2048", 64, 2048), ("decode 256 @2048", 256, 2048))


def kernels(out) -> None:
    import torch

    from omni_infer_b200 import ops
    from omni_infer_b200.ops import _native as nat
    from omni_infer_b200.ops import attention as A
    from omni_infer_b200.ops import attn_prepare as ap
    from omni_infer_b200.ops import layer_list as ll
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
        W, H, G, D, win, chunk = c["width"], c["heads"], c["kv_heads"], c["dim"], c["window"], c["chunk"]
        C, R, QR, eps = c["kv_rank"], c["rot_dim"], c["q_rank"], 1e-5
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
            seen_w, seen_c = min(win, L), L % chunk or min(chunk, L)
            pairs_w = B * (seen_w * (seen_w + 1) / 2 + (L - seen_w) * seen_w) if pre else B * seen_w
            full, rest = divmod(L, chunk)
            pairs_c = B * (full * chunk * (chunk + 1) / 2 + rest * (rest + 1) / 2) if pre else B * seen_c
            pairs = B * L * (L + 1) / 2 if pre else B * L
            # ---- residual and norm
            x, y, w1, b1, yr = f32(T, W), bf(T, W), torch.ones(W, device=dev), torch.zeros(W, device=dev), bf(T, W)
            wb = torch.ones(W, device=dev).bfloat16()
            row(size, what, "add_norm (bias)", lambda: ll.add_norm(x, y, w1, eps, torch.bfloat16, ld=W + 64, ones=True, bias=b1), T * W * 12)
            row(size, what, "  like: post_norm_add", lambda: ll.post_norm_add(y, w1, x, eps), T * W * 12)
            row(size, what, "  like: rmsnorm + residual", lambda: ops.rmsnorm(y, wb, eps, residual=yr), T * W * 8)
            # ---- windowed and chunked attention
            n = (H + 2 * G) * D
            wq, wq0, h1, h0 = bf(n, W + 64), bf(n, W), bf(T, W + 64), bf(T, W)
            row(size, what, "qkv gemm, biases as a column", lambda: ops.gemm(h1, wq), (n * W + T * W + T * n) * 2, 2.0 * T * W * n)
            row(size, what, "  like: qkv gemm", lambda: ops.gemm(h0, wq0), (n * W + T * W + T * n) * 2, 2.0 * T * W * n)
            del wq, wq0, h1
            kc, vc = bf(B * nblk + 1, bs, G, D), bf(B * nblk + 1, bs, G, D)
            qkv, first, lam = bf(T, n), bf(T, n), torch.full((1,), 0.4, device=dev)
            cs = ops.rope_cos_sin_table(D, 8200, 5e5, None, device=dev)
            qn, qnb = torch.ones(D, device=dev), torch.ones(D, device=dev).bfloat16()
            row(size, what, "qkv_prepare (norm, rotation, mix)",
                lambda: ap.qkv_prepare(qkv, H, G, D, D, qn, qn, eps, cs, D, True, pos, slots, kc, vc, mix=lam, v_first=first[:, (H + G) * D:]),
                T * ((H + G) * 2 + 3 * G) * D * 2)
            row(size, what, "qkv_prepare (cache write, mix)",
                lambda: ap.qkv_prepare(qkv, H, G, D, D, None, None, eps, None, 0, False, pos, slots, kc, vc, mix=lam, v_first=first[:, (H + G) * D:]),
                T * 5 * G * D * 2)
            row(size, what, "  like: rope_qk_cache (per-head norm)", lambda: ops.rope_qk_cache(qkv, H, G, D, cs, pos, slots, kc, vc, qnb, qnb, eps),
                T * ((H + G) * 2 + 2 * G) * D * 2)
            cw, cst = f32(c["conv"], n), torch.zeros(B, c["conv"] - 1, n, device=dev).bfloat16()
            p1 = pos if pre else torch.full_like(pos, L)
            where = dict(positions=p1, state_slots=ss, q_to_seq=seq, cu_q=cq)
            by = (2 * T * n + 2 * B * (c["conv"] - 1) * n) * 2
            row(size, what, "short_conv of q, k, v", lambda: ll.short_conv(qkv, cw, None, cst, **where), by)
            cb = f32(n)
            row(size, what, "  like: conv_silu", lambda: ll.conv_silu(qkv, cw, cb, cst, **where), by)
            qkv = bf(T, n)
            q3 = qkv[:, : H * D].unflatten(1, (H, D))
            slopes = 2.0 ** (-8.0 * torch.arange(1, H + 1, device=dev) / H)
            kw = dict(positions=pos, q_to_seq=seq, slots=slots, block_table=bt, seq_lens=sl, scale=D ** -0.5, cu_q=cq, max_q=T // B, max_seq_len=L)
            io = lambda seen: T * (2 * H + 2 * G) * D * 2 if pre else (B * seen * 2 * G + 2 * B * H) * D * 2      # noqa: E731
            row(size, what, f"attention, window {win} + {c['keep_first']} kept",
                lambda: ll.paged_attention(q3, kc, vc, window=win, keep_first=c["keep_first"], **kw), io(seen_w), pairs_w * H * 4 * D)
            row(size, what, f"attention, chunks of {chunk}, capped, biased",
                lambda: ll.paged_attention(q3, kc, vc, chunk=chunk, softcap=30.0, slopes=slopes, **kw), io(seen_c), pairs_c * H * 4 * D)
            row(size, what, "attention, capped, biased (all keys)", lambda: ll.paged_attention(q3, kc, vc, softcap=30.0, slopes=slopes, **kw),
                io(L), pairs * H * 4 * D)
            if pre:
                k3, v3 = qkv[:, H * D:(H + G) * D].unflatten(1, (G, D)), qkv[:, (H + G) * D:].unflatten(1, (G, D))
                row(size, what, "  like: gqa_prefill", lambda: A.gqa_prefill(q3, k3, v3, cu, cu, D ** -0.5, L, L), io(L), pairs * H * 4 * D)
            else:
                qc = q3.contiguous()
                row(size, what, "  like: gqa_decode", lambda: A.gqa_decode(qc, kc, vc, bt, sl, D ** -0.5, L), io(L), pairs * H * 4 * D)
            del kc, vc, qkv, q3, first
            # ---- latent attention
            ld = QR + C + R + H
            a, cache = bf(T, ld), bf(B * nblk + 1, bs, C + R)
            csr = ops.rope_cos_sin_table(R, 8200, 1e4, None, device=dev)
            qw, cw = torch.ones(QR, device=dev), torch.ones(C, device=dev)
            row(size, what, "latent_prepare", lambda: ap.latent_prepare(a, QR, QR, C, R, qw, cw, eps, csr, pos, slots, cache, C, QR, pre),
                T * ((QR + C + R) * 2 + (C + R) * pre) * 2)
            q, cwb, qwb = bf(T, H, D + R), cw.bfloat16(), qw.bfloat16()
            row(size, what, "rotate_heads", lambda: ap.rotate_heads(q[..., D:], R, csr, pos, q[..., D:]), T * H * R * 4)
            row(size, what, "  like: rmsnorm of the query latent", lambda: ops.rmsnorm(a[:, :QR], qwb, eps), T * QR * 4)
            row(size, what, "  like: mla_kv_rope_cache",
                lambda: ops.mla_kv_rope_cache(a[:, QR:QR + C + R], cwb, eps, csr, pos, slots, cache, q=q, q_rope_off=D, want_latent=pre),
                T * ((C + R) * (2 + pre) + 2 * H * R) * 2)
            gate = a[:, QR + C + R:]
            if pre:
                rows_, wkv = bf(T, C + R), bf(H * 2 * D, C)
                row(size, what, "key and value gemm", lambda: ops.gemm(rows_[:, :C], wkv), (T * (C + H * 2 * D) + H * 2 * D * C) * 2, 4.0 * T * H * D * C)
                kv = ops.gemm(rows_[:, :C], wkv)
                s0, s1 = cu[:-1], cu[1:]
                seg = dict(d1=D, dv=D, q_start=s0, q_end=s1, k_start=s0, k_end=s1, max_q=L, scale=(D + R) ** -0.5)
                by = T * (H * (D + R + 2 * D + D) + R) * 2
                fl = H * 2.0 * (D + R + D)
                row(size, what, f"latent_prefill, window {win}, gates", lambda: ap.latent_prefill(q, kv, rows_[:, C:], window=win, gate=gate, **seg), by,
                    pairs_w * fl)
                row(size, what, "latent_prefill, gates (all keys)", lambda: ap.latent_prefill(q, kv, rows_[:, C:], gate=gate, **seg), by, pairs * fl)
                row(size, what, "  like: mla_prefill", lambda: A.mla_prefill(q, kv, rows_, H, D, R, D, cu, cu, (D + R) ** -0.5, L, L), by, pairs * fl)
                i0 = torch.zeros(B, dtype=torch.int32, device=dev)
                row(size, what, "gather_pages", lambda: ap.gather_pages(cache, bt, ss, i0, s0, s1, T, L), T * (C + R) * 4)
                del rows_, wkv, kv
            else:
                qa = bf(T, H, C + R)
                lat = dict(positions=pos, q_to_seq=seq, slots=slots, block_table=bt, seq_lens=sl, scale=(D + R) ** -0.5, max_seq_len=L)
                io = lambda s: (B * s * (C + R) + T * H * (2 * C + R)) * 2      # noqa: E731
                fl = H * 2.0 * (2 * C + R)
                row(size, what, f"latent_attention, window {win}, gates", lambda: ap.latent_attention(qa, cache, C, window=win, gate=gate, **lat),
                    io(seen_w), B * seen_w * fl)
                row(size, what, "latent_attention, gates (all keys)", lambda: ap.latent_attention(qa, cache, C, gate=gate, **lat), io(L), B * L * fl)
                row(size, what, "  like: mla_decode", lambda: ops.mla_decode(qa, cache, bt, sl, (D + R) ** -0.5, max_seq_len=L), io(L), B * L * fl)
                del qa
            del a, cache, q
            # ---- experts
            E, k, ff = c["experts"], c["top"], c["expert_ff"]
            wr, bias = bf(E, W) * 0.1, torch.zeros(E, device=dev)
            lg = ops.gemm(h0, wr, out_dtype=torch.float32)
            row(size, what, "router_topk (bias, softmax of the chosen)", lambda: ops.router_topk(lg, k, renorm=True, logit_bias=bias), T * (E + 2 * k) * 4)
            row(size, what, "  like: router_topk", lambda: ops.router_topk(lg, k, renorm=True), T * (E + 2 * k) * 4)
            ids, wt = ops.router_topk(lg, k, renorm=True, logit_bias=bias)
            pm = ops.moe_permute(h0, ids, wt, 0, E)
            used, n_rows = int((pm.seg_len > 0).sum()), int(pm.seg_len.sum())
            w13, w2 = bf(E, 2 * ff, W), bf(E, W, ff)
            seg = dict(seg_start=pm.seg_start, seg_len=pm.seg_len, t_hint=max(16, (T * k + E - 1) // E))
            row(size, what, "grouped gemm + swiglu (the same kernel)", lambda: ops.gemm(pm.x, w13, epi="swiglu", **seg),
                (used * 2 * ff * W + n_rows * (W + ff)) * 2, 4.0 * n_rows * W * ff)
            act = ops.gemm(pm.x, w13, epi="swiglu", **seg)
            ye = ops.gemm(act, w2, row_scale=pm.row_w, **seg)
            es = st.ExpertSum(ye, pm.row_of, ids, wt, E, h0, y)
            row(size, what, "add_norm + expert sum", lambda: ll.add_norm(x, es, w1, eps, torch.bfloat16, ld=W), T * W * 12 + n_rows * W * 2)
            row(size, what, "  like: moe_combine", lambda: ops.moe_combine(ye, pm.row_of, T, k, shared=y), T * W * 4 + n_rows * W * 2)
            del w13, w2, x, ye, act, pm
            # ---- dense feed-forward
            F = c["ff"]
            wgu, h1 = bf(2 * F, W + 64), bf(T, W + 64)
            by, fl = (2 * F * W + T * W + T * F) * 2, 4.0 * T * W * F
            row(size, what, "gemm + swiglu, biases as a column", lambda: ops.gemm(h1, wgu, epi="swiglu"), by, fl)
            del wgu
            wgu = bf(2 * F, W)
            row(size, what, "  like: gemm + swiglu", lambda: ops.gemm(h0, wgu, epi="swiglu"), by, fl)
            del wgu, h1, h0
            torch.cuda.empty_cache()


def mla_like(c, **kw):
    """The MLA expert model (DeepSeek-V3 architecture) at the sizes ``c``."""
    from omni_infer_b200.models.config import ModelConfig
    return ModelConfig(architecture="DeepseekV3ForCausalLM", name="mla-moe", num_key_value_heads=c["heads"], q_lora_rank=c.get("q_rank", 0),
                       kv_lora_rank=c["kv_rank"], qk_nope_head_dim=c["dim"], qk_rope_head_dim=c["rot_dim"], v_head_dim=c["dim"],
                       n_shared_experts=c["shared_ff"] // c["expert_ff"], first_k_dense_replace=1, **_common(c), **kw)


def qwen_like(c):
    """The GQA expert model (Qwen3-MoE architecture) at the sizes ``c``."""
    from omni_infer_b200.models.config import ModelConfig
    return ModelConfig(architecture="Qwen3MoeForCausalLM", name="qwen3-moe", num_key_value_heads=c["kv_heads"], head_dim=c["dim"],
                       use_mla=False, n_shared_experts=0, first_k_dense_replace=0, qk_norm=True, rope_theta=1e6, **_common(c))


def _common(c):
    return dict(vocab_size=c["vocab"], hidden_size=c["width"], num_hidden_layers=c["layers"], num_attention_heads=c["heads"],
                intermediate_size=c["ff"], moe_intermediate_size=c["expert_ff"], n_routed_experts=c["experts"],
                num_experts_per_tok=c["top"], scoring_func="softmax", topk_method="greedy", norm_topk_prob=True,
                max_position_embeddings=9216)


def models(out) -> None:
    from omni_infer_b200.models.config import tenotar
    for size, c in SIZES.items():
        for name, mc in (("tenotar", tenotar(**c)), ("mla-moe", mla_like(c)), ("qwen3-moe", qwen_like(c))):
            throughput(out, size, c, name, mc)


def throughput(out, size, c, name, mc, steps=20, warmup=5) -> None:
    """Prefill and decode of a whole model through the engine."""
    import torch

    from omni_infer_b200.engine.engine_core import EngineConfig, EngineCore
    from omni_infer_b200.engine.request import SamplingParams
    from omni_infer_b200.ops import _native as nat

    for B, L in ((64, 1024), (256, 1024)):
        per = L + steps + warmup + 16
        eng = EngineCore(EngineConfig(model=name, block_size=128, num_kv_blocks=B * ((per + 127) // 128 + 1) + 1, max_num_seqs=B,
                                      max_num_batched_tokens=8192, max_model_len=per + 128, decode_gear_list=[B]), model_cfg=mc)
        g = torch.Generator().manual_seed(1)
        prompts = torch.randint(0, c["vocab"], (B, L), generator=g)
        sp = SamplingParams(max_tokens=10 ** 6, ignore_eos=True)
        for p in prompts:
            eng.add_request(p.tolist(), sp)
        ts = []
        while eng.scheduler.num_waiting:
            n0 = eng.scheduler.stats["scheduled_prefill_tokens"]
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            eng.step()
            b.record()
            torch.cuda.synchronize()
            ts.append((eng.scheduler.stats["scheduled_prefill_tokens"] - n0, a.elapsed_time(b)))
        ts = ts[2:] if len(ts) > 4 else ts[1:]
        n_tok, ms = sum(t[0] for t in ts), sum(t[1] for t in ts)
        for _ in range(warmup):
            eng.step()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(steps):
            eng.step()
        b.record()
        torch.cuda.synchronize()
        nat.check_status()
        dec = a.elapsed_time(b) / steps
        nparam = sum(p.numel() for p in eng.worker.runner.model.parameters())
        out({"size": size, "model": name, "layers": c["layers"], "params_M": round(nparam / 1e6), "batch": B, "prompt": L,
             "prefill_tok_s": round(n_tok / ms * 1e3), "decode_ms_per_step": round(dec, 3), "decode_tok_s": round(B / dec * 1e3),
             "cuda_graph": eng.worker.runner.graphs is not None})
        del eng
        torch.cuda.empty_cache()


def main(which: str) -> int:
    def out(d):
        print(json.dumps(d), flush=True)
    if which in ("tenotar-kernels", "tenotar"):
        kernels(out)
    if which in ("tenotar-model", "tenotar"):
        models(out)
    return 0

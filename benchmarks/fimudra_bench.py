#!/usr/bin/env python
"""The Fimudra design (residual streams, attention with a sink beside a matrix memory, WKV, clamped expert mixtures) beside the
framework's closest models at equal sizes, random weights.

    python bench.py --layer-list fimudra-kernels    each kernel against its roofline, beside the like kernel of the other models
    python bench.py --layer-list fimudra-model      prefill and decode throughput through the engine, beside a GQA expert model
    python bench.py --layer-list fimudra            both

Timing as in ``layer_list_bench.py``."""
from __future__ import annotations

import json

from .layer_list_bench import PEAKS, Timer

# width, attention heads / kv heads / size, matrix memory heads / key / value size, WKV heads / size / rank, experts, top, ff
SIZES = {
    "2k": dict(width=2048, layers=12, heads=16, kv_heads=4, dim=128, m_heads=16, m_dim=64, m_vdim=128, w_heads=32, w_dim=64, w_rank=64,
               experts=32, identity=4, top=4, ff=768, shared_ff=1536, streams=2, vocab=32768),
    "4k": dict(width=4096, layers=6, heads=32, kv_heads=8, dim=128, m_heads=16, m_dim=128, m_vdim=256, w_heads=64, w_dim=64, w_rank=128,
               experts=64, identity=8, top=6, ff=1024, shared_ff=2048, streams=4, vocab=32768),
}
CASES = (("prefill 8x1024", 8, 1024), ("prefill 1x8192", 1, 8192), ("decode 64 @2048", 64, 2048), ("decode 256 @2048", 256, 2048))


def kernels(out) -> None:
    import torch

    from omni_infer_b200 import ops
    from omni_infer_b200.ops import _native as nat
    from omni_infer_b200.ops import attention as A
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
        W, S, H, G, D = c["width"], c["streams"], c["heads"], c["kv_heads"], c["dim"]
        eps = 1e-5
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
            rec = dict(positions=pos, state_slots=ss, cu_q=cq)
            span = dict(min_q=T // B, max_q=T // B)
            # ---- residual streams: fp32 streams read and written, sublayer output read, next input written
            x, y, w1 = f32(T, S, W), bf(T, W), torch.ones(W, device=dev)
            mix, vec = f32(S, S) * 0.1 + torch.eye(S, device=dev), torch.ones(S, device=dev)
            row(size, what, f"stream_step ({S} streams)", lambda: st.stream_step(x, y, mix, vec, vec, w1, eps, torch.bfloat16),
                T * W * (8 * S + 4))
            xr, yr = f32(T, W), bf(T, W)
            row(size, what, "  like: post_norm_add", lambda: ll.post_norm_add(yr, w1, xr, eps), T * W * 12)
            del x, xr
            # ---- attention with a sink
            kc, vc = bf(B * nblk + 1, bs, G, D), bf(B * nblk + 1, bs, G, D)
            qkv, sink = bf(T, (H + 2 * G) * D), f32(H)
            cs = ops.rope_cos_sin_table(D, 8200, 5e5, None, device=dev)
            row(size, what, "rotation + cache write", lambda: ll.qk_norm_rope_cache(qkv, H, G, D, D, None, None, eps, cs, D, pos, slots, kc, vc),
                T * ((H + G) * 2 + 2 * G) * D * 2)
            qnb, knb = torch.ones(D, device=dev).bfloat16(), torch.ones(D, device=dev).bfloat16()
            row(size, what, "  like: rope_qk_cache (per-head norm)",
                lambda: ops.rope_qk_cache(qkv, H, G, D, cs, pos, slots, kc, vc, qnb, knb, eps), T * ((H + G) * 2 + 2 * G) * D * 2)
            qkv = bf(T, (H + 2 * G) * D)
            q3 = qkv[:, : H * D].unflatten(1, (H, D))
            fl = (B * L * (L + 1) / 2 if pre else B * L) * H * 4 * D
            by = T * (2 * H + 2 * G) * D * 2 if pre else (B * L * 2 * G + 2 * B * H) * D * 2
            row(size, what, "paged_attention with a sink",
                lambda: ll.paged_attention(q3, kc, vc, positions=pos, q_to_seq=seq, slots=slots, block_table=bt, seq_lens=sl, scale=D ** -0.5,
                                           cu_q=cq, max_q=T // B, max_seq_len=L, sink=sink, out_scale=0.7), by, fl)
            if pre:
                k3, v3 = qkv[:, H * D:(H + G) * D].unflatten(1, (G, D)), qkv[:, (H + G) * D:].unflatten(1, (G, D))
                row(size, what, "  like: gqa_prefill", lambda: A.gqa_prefill(q3, k3, v3, cu, cu, D ** -0.5, L, L), by, fl)
            else:
                qc = q3.contiguous()
                row(size, what, "  like: gqa_decode", lambda: A.gqa_decode(qc, kc, vc, bt, sl, D ** -0.5, L), by, fl)
            del kc, vc, qkv, q3
            # ---- matrix memory
            MH, N, P = c["m_heads"], c["m_dim"], c["m_vdim"]
            u, z = bf(T, MH * (2 * N + 2 * P)), f32(T, 2 * MH)
            ib, fb = f32(MH), f32(MH) + 3
            Sm, m = torch.zeros(B, MH, P + 1, N, device=dev), torch.zeros(B, MH, device=dev)
            p1 = pos if pre else torch.full_like(pos, L)
            rec1 = dict(rec, positions=p1)
            chunks = pre and ms.mlstm_chunked(torch.bfloat16, N, P)
            gates = ms.mlstm_gates(z, MH, ib, fb, 15.0, m, chunks=chunks, **rec1)
            row(size, what, "mlstm_gates", lambda: ms.mlstm_gates(z, MH, ib, fb, 15.0, m, chunks=chunks, **rec1), T * MH * (8 + 16 + 12 * pre))
            q_, k_, v_, g_ = u[:, :MH * N], u[:, MH * N:2 * MH * N], u[:, 2 * MH * N:MH * (2 * N + P)], u[:, MH * (2 * N + P):]
            fl = T * MH * (64 * (N + P) + 4.0 * N * P) if pre else 0
            by = T * MH * (2 * N + 2 * P) * 2 + B * MH * (P + 1) * N * 4 * (1 if pre else 2)
            row(size, what, "mlstm_scan", lambda: ms.mlstm_scan(q_, k_, v_, gates, Sm, H=MH, P=P, N=N, **rec1, **span), by, fl)
            xbc, dt = bf(T, MH * (P + 2 * N)), bf(T, MH)
            A_log, dtb, Dv, ssm = f32(MH) * 0.5, f32(MH) * 0.5 - 3, f32(MH), torch.zeros(B, MH, P, N, device=dev)
            row(size, what, "  like: ssm_scan (beside mlstm)",
                lambda: ll.ssm_scan(xbc, dt, A_log, dtb, Dv, ssm, H=MH, P=P, N=N, G=MH, **rec1, **span), by, fl)
            yy, nw, oo = bf(T, MH * P), torch.ones(MH * P, device=dev), bf(T, MH * P)
            row(size, what, "head_norm (matrix memory)", lambda: ms.head_norm(yy, g_, nw, oo, H=MH, P=P, eps=eps, act="sigmoid", gates=gates),
                T * MH * P * 6)
            row(size, what, "  like: gated_group_norm (beside matrix memory)", lambda: ll.gated_group_norm(yy, oo, nw, MH, eps), T * MH * P * 6)
            del u, xbc, Sm, ssm
            # ---- WKV
            WH, ND, R = c["w_heads"], c["w_dim"], c["w_rank"]
            n = WH * ND
            mu, last, h = torch.rand(5, W, device=dev), torch.zeros(B, W, device=dev).bfloat16(), bf(T, W)
            row(size, what, "token_shift (5 mixes)", lambda: st.token_shift(h, mu, last, W, q_to_seq=seq, **rec1), T * W * 12)
            cw, cb, cst = f32(4, W), f32(W), torch.zeros(B, 3, W, device=dev).bfloat16()
            row(size, what, "  like: conv_silu", lambda: ll.conv_silu(h, cw, cb, cst, q_to_seq=seq, **rec1), (2 * T * W + 6 * B * W) * 2)
            xs, w4 = bf(T, 5, W), bf(4, n, W)
            row(size, what, "r k v g grouped gemm", lambda: ops.bmm_heads(xs[:, :4], w4), (4 * n * W + T * 4 * (W + n)) * 2, 8.0 * T * W * n)
            wq = w4.view(4 * n, W)
            row(size, what, "  like: gemm of that size", lambda: ops.gemm(h, wq), (4 * n * W + T * W + T * 4 * n) * 2, 8.0 * T * W * n)
            w1_, w2_ = bf(R, W), bf(n, 2 * R)
            row(size, what, "decay projections (3 kernels)",
                lambda: ops.gemm(st.tanh_split(ops.gemm(xs[:, 4], w1_, out_dtype=torch.float32), R, torch.bfloat16), w2_, out_dtype=torch.float32),
                (T * W + R * W + 2 * n * R) * 2 + T * (R * 12 + n * 4), 2.0 * T * R * (W + 2 * n))
            del w4, wq
            pr, zz = bf(T, 4, n), f32(T, n)
            w0, uu, Sw = f32(n), f32(n), torch.zeros(B, WH, ND, ND, device=dev)
            fl = T * WH * (64 * 2 * ND + 4.0 * ND * ND) if pre else 0
            by = T * n * 12 + B * WH * ND * ND * 4 * (1 if pre else 2)
            row(size, what, "wkv_scan", lambda: ms.wkv_scan(pr[:, 0], pr[:, 1], pr[:, 2], zz, w0, uu, Sw, H=WH, N=ND, **rec1, **span), by, fl)
            xbc, dt = bf(T, 3 * n), bf(T, WH)
            A_log, dtb, Dv = f32(WH) * 0.5, f32(WH) * 0.5 - 3, f32(WH)
            by = T * n * 8 + B * WH * ND * ND * 4 * (1 if pre else 2)
            row(size, what, "  like: ssm_scan (beside wkv)",
                lambda: ll.ssm_scan(xbc, dt, A_log, dtb, Dv, Sw, H=WH, P=ND, N=ND, G=WH, **rec1, **span), by, fl)
            yy, nw, oo = bf(T, n), torch.ones(n, device=dev), bf(T, n)
            row(size, what, "head_norm (WKV)", lambda: ms.head_norm(yy, pr[:, 3], nw, oo, H=WH, P=ND, eps=eps, act="silu"), T * n * 6)
            row(size, what, "  like: gated_group_norm (beside WKV)", lambda: ll.gated_group_norm(yy, oo, nw, WH, eps), T * n * 6)
            del xbc, pr, zz, xs
            # ---- experts
            E, I, k, ff = c["experts"], c["identity"], c["top"], c["ff"]
            wr, bias = bf(E + I, W) * 0.1, torch.zeros(E + I, device=dev)
            lg = ops.gemm(h, wr, out_dtype=torch.float32)
            row(size, what, "router gemm", lambda: ops.gemm(h, wr, out_dtype=torch.float32), (T * W + (E + I) * W) * 2 + T * (E + I) * 4)
            ids, wt = ops.router_topk(lg, k, mode="softmax", bias=bias, scale=2.5)
            row(size, what, "router_topk", lambda: ops.router_topk(lg, k, mode="softmax", bias=bias, scale=2.5), T * (E + I + 2 * k) * 4)
            row(size, what, "moe_permute", lambda: ops.moe_permute(h, ids, wt, 0, E), T * W * 2 + T * k * W * 2)
            pm = ops.moe_permute(h, ids, wt, 0, E)
            used = int((pm.seg_len > 0).sum())
            n_rows = int(pm.seg_len.sum())
            w13, w2 = bf(E, 2 * ff, W), bf(E, W, ff)
            kw = dict(seg_start=pm.seg_start, seg_len=pm.seg_len, t_hint=max(16, (T * k + E - 1) // E))
            by, fl = (used * 2 * ff * W + n_rows * (W + ff)) * 2, 4.0 * n_rows * W * ff
            row(size, what, "grouped gemm + clamped glu", lambda: ops.gemm(pm.x, w13, epi="clamped_glu", glu_limit=7.0, **kw), by, fl)
            row(size, what, "  like: grouped gemm + swiglu", lambda: ops.gemm(pm.x, w13, epi="swiglu", **kw), by, fl)
            act = ops.gemm(pm.x, w13, epi="clamped_glu", glu_limit=7.0, **kw)
            row(size, what, "grouped gemm (down)", lambda: ops.gemm(act, w2, row_scale=pm.row_w, **kw), (used * ff * W + n_rows * (W + ff)) * 2,
                2.0 * n_rows * W * ff)
            ye = ops.gemm(act, w2, row_scale=pm.row_w, **kw)
            x = f32(T, S, W)
            es = st.ExpertSum(ye, pm.row_of, ids, wt, E, h, y)
            row(size, what, "stream_step + expert sum", lambda: st.stream_step(x, es, mix, vec, vec, w1, eps, torch.bfloat16),
                T * W * (8 * S + 2 + 4) + n_rows * W * 2)
            row(size, what, "  like: moe_combine", lambda: ops.moe_combine(ye, pm.row_of, T, k, shared=y), T * W * 4 + n_rows * W * 2)
            del w13, w2, x, ye, act, pm
            torch.cuda.empty_cache()


def models(out, steps=20, warmup=5) -> None:
    import torch

    from omni_infer_b200.engine.engine_core import EngineConfig, EngineCore
    from omni_infer_b200.engine.request import SamplingParams
    from omni_infer_b200.models.config import ModelConfig, fimudra
    from omni_infer_b200.ops import _native as nat

    def qwen(c):
        return ModelConfig(architecture="Qwen3MoeForCausalLM", name="qwen3-moe", vocab_size=c["vocab"], hidden_size=c["width"],
                           num_hidden_layers=c["layers"], num_attention_heads=c["heads"], num_key_value_heads=c["kv_heads"],
                           head_dim=c["dim"], use_mla=False, intermediate_size=c["shared_ff"], moe_intermediate_size=c["ff"],
                           n_routed_experts=c["experts"], n_shared_experts=0, num_experts_per_tok=c["top"], first_k_dense_replace=0,
                           scoring_func="softmax", topk_method="greedy", norm_topk_prob=True, qk_norm=True, rope_theta=1e6,
                           max_position_embeddings=9216)

    for size, c in SIZES.items():
        for name, mc in (("fimudra", fimudra(loop=False, **c)), ("qwen3-moe", qwen(c))):
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
    if which in ("fimudra-kernels", "fimudra"):
        kernels(out)
    if which in ("fimudra-model", "fimudra"):
        models(out)
    return 0

#!/usr/bin/env python
"""Layer-list models (windowed attention + Mamba-2) beside the framework's GQA model at equal sizes, random weights.

    python bench.py --layer-list kernels        each kernel against its roofline, beside the like kernel of the GQA model
    python bench.py --layer-list model          prefill and decode throughput of whole models through the engine
    python bench.py --layer-list all

Kernel times are CUDA events around a captured graph of one call, L2 flushed before every iteration (a 256 MB write that is
still running while the next call is queued, so host time does not show).  "roofline" is the larger of algorithmic bytes
over the measured copy bandwidth and algorithmic FLOPs over the measured cuBLAS bf16 throughput, divided by the time."""
from __future__ import annotations

import json
import os
import statistics
import sys
import time

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

PEAKS = {"hbm_gbs": 6533.2, "bf16_tflops": 1657.8}
try:
    PEAKS.update(json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json"))))
except Exception:  # noqa: BLE001
    pass

# width, layers, attention heads, kv heads, head size, window, ff, Mamba-2 heads, head size, state, groups
SIZES = {
    "2k": dict(width=2048, layers=12, heads=16, kv_heads=4, dim=128, window=1024, ff=5632, m_heads=64, m_vdim=64, state=128,
               groups=1, vocab=32768),
    "4k": dict(width=4096, layers=6, heads=32, kv_heads=8, dim=128, window=1024, ff=11264, m_heads=128, m_vdim=64, state=128,
               groups=8, norm_groups=8, vocab=32768),
}


class Timer:
    def __init__(self, iters=15, warm=3):
        import torch
        self.torch, self.iters, self.warm = torch, iters, warm
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def __call__(self, fn) -> float:
        torch = self.torch
        s = torch.cuda.Stream()
        s.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(s):
            for _ in range(2):
                fn()
        torch.cuda.current_stream().wait_stream(s)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            fn()
        ts = []
        for i in range(self.warm + self.iters):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            self.flush.fill_(i & 1)
            a.record()
            g.replay()
            b.record()
            torch.cuda.synchronize()
            if i >= self.warm:
                ts.append(a.elapsed_time(b) * 1e3)
        return statistics.median(ts)


def kernels(out) -> None:
    import torch

    from omni_infer_b200 import ops
    from omni_infer_b200.ops import _native as nat
    from omni_infer_b200.ops import attention as A
    from omni_infer_b200.ops import layer_list as ll
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

    def pages(B, ctx, bs=128):
        nb = (ctx + bs - 1) // bs
        return torch.arange(1, B * nb + 1, dtype=torch.int32, device=dev).view(B, nb), B * nb + 1, bs

    for size, c in SIZES.items():
        W, H, G, D, ff = c["width"], c["heads"], c["kv_heads"], c["dim"], c["ff"]
        MH, P, N, MG = c["m_heads"], c["m_vdim"], c["state"], c["groups"]
        inner, C = MH * P, MH * P + 2 * MG * N
        qkv_n = (H + 2 * G) * D
        eps, scale = 1e-5, D ** -0.5
        cs = ops.rope_cos_sin_table(D, 8200, 1e6, None, device=dev)
        w_small = torch.ones(W, device=dev)
        for what, B, L in (("prefill 8x1024", 8, 1024), ("prefill 1x8192", 1, 8192), ("decode 64 @2048", 64, 2048),
                           ("decode 256 @2048", 256, 2048)):
            pre = what.startswith("prefill")
            T = B * L if pre else B
            bt, nb, bs = pages(B, L)
            kc, vc = bf(nb, bs, G, D), bf(nb, bs, G, D)
            pos = (torch.arange(L, device=dev).repeat(B) if pre else torch.full((B,), L - 1, device=dev)).contiguous()
            seq = torch.arange(B, dtype=torch.int32, device=dev).repeat_interleave(T // B)
            slots = bt[seq.long(), pos // bs].long() * bs + pos % bs
            cu = torch.arange(B + 1, dtype=torch.int32, device=dev) * (T // B)
            sl = torch.full((B,), L, dtype=torch.int32, device=dev)
            cq = cu if pre else None
            # ---- row kernels
            y, x, res = bf(T, W), f32(T, W), bf(T, W)
            row(size, what, "post_norm_add", lambda: ll.post_norm_add(y, w_small, x, eps), T * W * 12)
            wb = torch.ones(W, device=dev).bfloat16()
            row(size, what, "  like: rmsnorm + residual", lambda: ops.rmsnorm(y, wb, eps, residual=res), T * W * 8)
            qkv = bf(T, qkv_n)
            qn, kn = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
            row(size, what, "qk_norm_rope_cache", lambda: ll.qk_norm_rope_cache(qkv, H, G, D, D, qn, kn, eps, cs, D, pos, slots, kc, vc),
                T * qkv_n * 4)
            qnb, knb = torch.ones(D, device=dev).bfloat16(), torch.ones(D, device=dev).bfloat16()
            row(size, what, "  like: rope_qk_cache (per-head norm)",
                lambda: ops.rope_qk_cache(qkv, H, G, D, cs, pos, slots, kc, vc, qnb, knb, eps), T * (qkv_n + (H + 2 * G) * D) * 2)
            # ---- attention
            qkv = bf(T, qkv_n)      # the timed kernels above have normed theirs over and over
            q3 = qkv[:, : H * D].unflatten(1, (H, D))
            kw = dict(positions=pos, q_to_seq=seq, slots=slots, block_table=bt, seq_lens=sl, scale=scale, cu_q=cq,
                      max_q=T // B, max_seq_len=L)
            for win in (0, c["window"], 256):
                vis = min(win or L, L)
                if pre:
                    pairs = B * (vis * (vis + 1) / 2 + (L - vis) * vis)
                    fl, by = pairs * H * 4 * D, T * (2 * H + 2 * G) * D * 2
                else:
                    fl, by = B * vis * H * 4 * D, (B * vis * 2 * G + 2 * B * H) * D * 2
                row(size, what, f"paged_attention window {win}", lambda: ll.paged_attention(q3, kc, vc, window=win, **kw), by, fl)
            if pre:
                k3, v3 = qkv[:, H * D:(H + G) * D].unflatten(1, (G, D)), qkv[:, (H + G) * D:].unflatten(1, (G, D))
                row(size, what, "  like: gqa_prefill", lambda: A.gqa_prefill(q3, k3, v3, cu, cu, scale, L, L),
                    T * (2 * H + 2 * G) * D * 2, B * L * (L + 1) / 2 * H * 4 * D)
            else:
                qc = q3.contiguous()
                row(size, what, "  like: gqa_decode", lambda: A.gqa_decode(qc, kc, vc, bt, sl, scale, L),
                    (B * L * 2 * G + 2 * B * H) * D * 2, B * L * H * 4 * D)
            # ---- feed-forward
            wgu, xb = bf(2 * ff, W), bf(T, W)
            by, fl = (2 * ff * W + T * W + T * ff) * 2, 4.0 * T * W * ff
            row(size, what, "gemm + geglu", lambda: ops.gemm(xb, wgu, epi="geglu"), by, fl)
            row(size, what, "  like: gemm + swiglu", lambda: ops.gemm(xb, wgu, epi="swiglu"), by, fl)
            del wgu
            # ---- Mamba-2
            n_in = ll.pad8(inner + C + MH)
            win_, u = bf(n_in, W), bf(T, n_in)
            row(size, what, "in_proj gemm", lambda: ops.gemm(xb, win_), (n_in * W + T * W + T * n_in) * 2, 2.0 * T * W * n_in)
            wq = bf(qkv_n, W)
            row(size, what, "  like: qkv gemm", lambda: ops.gemm(xb, wq), (qkv_n * W + T * W + T * qkv_n) * 2, 2.0 * T * W * qkv_n)
            del win_, wq
            cw, cb = f32(4, C), f32(C)
            conv_state = torch.zeros(B, 3, C, device=dev, dtype=torch.bfloat16)
            ssm_state = torch.zeros(B, MH, P, N, device=dev)
            st = torch.arange(B, dtype=torch.int32, device=dev)
            p1 = pos if pre else torch.full_like(pos, L)
            row(size, what, "conv_silu", lambda: ll.conv_silu(u[:, inner:inner + C], cw, cb, conv_state, positions=p1, state_slots=st,
                                                              q_to_seq=seq, cu_q=cq), (2 * T * C + 2 * B * 3 * C) * 2)
            xbc = bf(T, C)
            A_log, dtb, Dv = f32(MH) * 0.5, f32(MH) * 0.5 - 3, f32(MH)
            chunk = 64
            fl = T * MH * (chunk * P + 4.0 * N * P) + T * MG * chunk * N if pre else 0
            by = T * (C + inner + MH) * 2 + B * MH * P * N * 4 * (1 if pre else 2)
            row(size, what, "ssm_scan", lambda: ll.ssm_scan(xbc, u[:, inner + C:inner + C + MH], A_log, dtb, Dv, ssm_state, H=MH, P=P,
                                                            N=N, G=MG, positions=p1, state_slots=st, cu_q=cq, min_q=T // B,
                                                            max_q=T // B), by, fl)
            yy, nw = bf(T, inner), torch.ones(inner, device=dev)
            row(size, what, "gated_group_norm", lambda: ll.gated_group_norm(yy, u, nw, c.get("norm_groups", 1), eps), T * inner * 6)
            del u, xbc, yy, kc, vc
            torch.cuda.empty_cache()


def models(out, steps=20, warmup=5) -> None:
    import torch

    from omni_infer_b200.engine.engine_core import EngineConfig, EngineCore
    from omni_infer_b200.engine.request import SamplingParams
    from omni_infer_b200.models.config import ModelConfig, forovik
    from omni_infer_b200.ops import _native as nat

    def qwen(c):
        return ModelConfig(architecture="Qwen2ForCausalLM", name="qwen2-dense", vocab_size=c["vocab"], hidden_size=c["width"],
                           num_hidden_layers=c["layers"], num_attention_heads=c["heads"], num_key_value_heads=c["kv_heads"],
                           head_dim=c["dim"], use_mla=False, intermediate_size=c["ff"], n_routed_experts=0, attention_bias=False,
                           rope_theta=1e6, max_position_embeddings=9216, tie_word_embeddings=True)

    for size, c in SIZES.items():
        for name, mc in (("forovik", forovik(**c)), ("qwen2-dense", qwen(c))):
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
                    t0 = time.perf_counter()
                    a.record()
                    eng.step()
                    b.record()
                    torch.cuda.synchronize()
                    ts.append((eng.scheduler.stats["scheduled_prefill_tokens"] - n0, a.elapsed_time(b), (time.perf_counter() - t0) * 1e3))
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
    if which in ("kernels", "all"):
        kernels(out)
    if which in ("model", "all"):
        models(out)
    return 0


if __name__ == "__main__":
    sys.exit(main(sys.argv[1] if len(sys.argv) > 1 else "all"))

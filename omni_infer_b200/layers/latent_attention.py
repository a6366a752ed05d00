"""Latent attention of the layer-list models: queries through a latent of their own or straight from the input, keys and values
projected from one cached latent per token, a rotated key part that all heads share, a sliding window or none, and optionally a
sigmoid gate per head and a sink per head in the softmax.

Single tokens (and fp32 runs, and head sizes that the kernel for portions does not take) attend in latent space: the key
projection is absorbed into the query and the value projection follows.  Portions of prompts project the latents of the keys
they can see - those of the step itself, or gathered from the pages.  Blocks of the weights are padded to multiples of 8 with
zeros, so all sizes can be TMA operands.

The kernels rotate dimension i together with i + rot_dim / 2.  Where neighbours turn together, the rows of the weights that make the
rotated parts are stored even ones first: queries and keys change alike, so their products stay."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..models.config import LatentSpec
from ..ops.attn_prepare import gather_pages, latent_attention, latent_prefill, latent_prefill_fits, latent_prepare, rotate_heads
from ..ops.layer_list import pad8
from .common import AttnMetadata, PaddedLinear

ABSORB_ROWS = 8      # requests with up to this many tokens in a step attend in latent space, too


@dataclass
class StepPlan:
    """Which requests of a ragged step take which form (device tensors int32 but for ``rows``)."""
    n_long: int
    n_short: int
    # long: query rows, key rows
    q_start: torch.Tensor = None
    q_end: torch.Tensor = None
    k_start: torch.Tensor = None
    k_end: torch.Tensor = None
    max_q: int = 0
    # keys that are not the step's own rows: which cached rows to gather
    gather: Optional[tuple] = None
    # short: rows of the step, their request and number of visible keys
    rows: torch.Tensor = None
    row_seq: torch.Tensor = None
    row_lens: torch.Tensor = None


def step_plan(md: AttnMetadata, window: int, device) -> StepPlan:
    """Made once per step and window size."""
    got = md.plans.get(("latent", window))
    if got is not None:
        return got
    long, short, at = [], [], 0
    for b, (n, ctx) in enumerate(zip(md.query_lens, md.context_lens)):
        (short if n <= ABSORB_ROWS else long).append((b, at, n, ctx))
        at += n
    p = StepPlan(len(long), len(short))
    dev = lambda v, dt=torch.int32: torch.tensor(v, dtype=dt).to(device, non_blocking=True)       # noqa: E731
    if long:
        starts, ends = [a for _, a, _, _ in long], [a + n for _, a, n, _ in long]
        p.max_q = max(n for _, _, n, _ in long)
        if all(ctx == 0 for _, _, _, ctx in long):
            p.q_start, p.q_end = p.k_start, p.k_end = dev([starts, ends])
        else:
            keys = [min(ctx, window - 1 if window else ctx) + n for _, _, n, ctx in long]
            k_end = torch.tensor(keys).cumsum(0).tolist()
            k_start = [e - k for e, k in zip(k_end, keys)]
            p.q_start, p.q_end, p.k_start, p.k_end, req, pos0 = dev(
                [starts, ends, k_start, k_end, [b for b, _, _, _ in long], [ctx + n - k for (_, _, n, ctx), k in zip(long, keys)]])
            p.gather = (req, pos0, k_end[-1], max(keys))
    if short:
        p.rows = dev([a + i for _, a, n, _ in short for i in range(n)], torch.int64)
        p.row_seq, p.row_lens = dev([[b for b, _, n, _ in short for _ in range(n)], [ctx + i + 1 for _, _, n, ctx in short for i in range(n)]])
    md.plans[("latent", window)] = p
    return p


class LatentAttention(nn.Module):
    out_bias = None
    ones = False

    def __init__(self, spec: LatentSpec, hidden: int, eps: float, *, dtype, device=None, cos_sin=None):
        super().__init__()
        self.spec, self.hidden, self.eps, self.cos_sin = spec, hidden, eps, cos_sin
        s = spec
        self.d, self.r, self.p, self.c = pad8(s.dim), s.rot_cols, pad8(s.vdim), s.latent_cols
        # rows of the input projection: query latent, or per head unrotated | rotated query | key/value latent, key part | gates,
        # each block from a multiple of 8 on
        self.kv0 = pad8(s.q_rank) if s.q_rank else s.heads * (self.d + self.r)
        self.g0 = self.kv0 + pad8(s.kv_rank + s.rot_dim)
        self.in_proj = PaddedLinear(hidden, self.g0 + (s.heads if s.gate else 0), dtype=dtype, device=device)
        par = lambda *n: nn.Parameter(torch.zeros(*n, dtype=dtype, device=device), requires_grad=False)       # noqa: E731
        one = lambda n: nn.Parameter(torch.ones(n, dtype=torch.float32, device=device), requires_grad=False)  # noqa: E731
        self.q_norm, self.kv_norm = one(s.q_rank) if s.q_rank else None, one(s.kv_rank)
        self.w_uq = par(s.heads * (self.d + self.r), pad8(s.q_rank)) if s.q_rank else None            # per head unrotated | rotated
        self.sink = nn.Parameter(torch.zeros(s.heads, dtype=torch.float32, device=device), requires_grad=False) if s.sink else None
        self.w_kv = par(s.heads * (self.d + self.p), self.c)                    # per head key | value
        self.o_proj = par(pad8(hidden), s.heads * self.p)
        self.w_uk = self.w_uv = None                                            # [H, c, d], [H, p, c] for the absorbed form

    @property
    def in_cols(self):
        return self.in_proj.in_features

    def _blocks(self):
        """Views by head of the padded weights: queries, keys and values, output."""
        s = self.spec
        q = self.w_uq.data if self.w_uq is not None else self.in_proj.weight.data[:self.kv0]
        return (q.view(s.heads, self.d + self.r, -1), self.w_kv.data.view(s.heads, self.d + self.p, -1),
                self.o_proj.data.view(-1, s.heads, self.p))

    def zero_padding(self):
        s = self.spec
        uq, kv, o = self._blocks()
        a = self.in_proj.weight.data
        if s.q_rank:
            a[s.q_rank:self.kv0] = 0
            uq[..., s.q_rank:] = 0
        a[self.kv0 + s.kv_rank + s.rot_dim:self.g0] = 0
        uq[:, s.dim:self.d] = 0
        uq[:, self.d + s.rot_dim:] = 0
        kv[:, s.dim:self.d] = 0
        kv[:, self.d + s.vdim:] = 0
        kv[..., s.kv_rank:] = 0
        o[self.hidden:] = 0
        o[..., s.vdim:] = 0
        self.w_uk = kv[:, :self.d].transpose(1, 2).contiguous()
        self.w_uv = kv[:, self.d:].contiguous()

    def forward(self, x, md: AttnMetadata, cache, shared=None):
        s, T = self.spec, x.shape[0]
        a = ops.gemm(x, self.in_proj.weight)
        portions = md.is_prefill and x.is_cuda and latent_prefill_fits(x.dtype, self.d, self.r, self.p, s.scale)
        plan = step_plan(md, s.window, x.device) if portions else None
        own_keys = portions and plan.n_long > 0 and plan.gather is None
        cq, rows = latent_prepare(a, s.q_rank, self.kv0, s.kv_rank, s.rot_dim, self.q_norm, self.kv_norm, self.eps, self.cos_sin,
                                  md.positions, md.slot_mapping, cache, self.c, pad8(s.q_rank), want_rows=own_keys)
        q = (ops.gemm(cq, self.w_uq) if s.q_rank else a[:, :self.kv0]).unflatten(1, (s.heads, self.d + self.r))
        gate = a[:, self.g0:self.g0 + s.heads] if s.gate else None
        if not portions:
            lens = md.q_seq_lens if not md.is_prefill else self._visible(md)
            o = self._absorbed(q, gate, md.positions, md.slot_mapping, md.q_to_seq, lens, md, cache)
        elif plan.n_long == 0:
            o = self._absorbed(q, gate, md.positions, md.slot_mapping, plan.row_seq, plan.row_lens, md, cache)
        else:
            part = None
            if plan.n_short:
                i = plan.rows
                part = self._absorbed(q[i], gate[i] if gate is not None else None, md.positions[i], md.slot_mapping[i], plan.row_seq,
                                      plan.row_lens, md, cache)
            rotate_heads(q[..., self.d:], s.rot_dim, self.cos_sin, md.positions, q[..., self.d:])
            if plan.gather is not None:
                req, pos0, total, longest = plan.gather
                rows = gather_pages(cache, md.block_table, req, pos0, plan.k_start, plan.k_end, total, longest)
            kv = ops.gemm(rows[:, :self.c], self.w_kv)
            o = latent_prefill(q, kv, rows[:, self.c:], d1=self.d, dv=self.p, q_start=plan.q_start, q_end=plan.q_end, k_start=plan.k_start,
                               k_end=plan.k_end, max_q=plan.max_q, scale=s.scale, window=s.window, gate=gate, sink=self.sink)
            if part is not None:
                o[plan.rows] = part
        return ops.gemm(o, self.o_proj)

    @staticmethod
    def _visible(md):
        """Visible keys of every row of a ragged step."""
        if "visible" not in md.plans:
            md.plans["visible"] = (md.positions + 1).int()
        return md.plans["visible"]

    def _absorbed(self, q, gate, positions, slots, q_to_seq, lens, md, cache):
        s, T = self.spec, q.shape[0]
        qa = torch.empty(T, s.heads, self.c + self.r, dtype=q.dtype, device=q.device)
        ops.bmm_heads(q[..., :self.d], self.w_uk, out=qa)
        rotate_heads(q[..., self.d:], s.rot_dim, self.cos_sin, positions, qa[..., self.c:])
        lat = latent_attention(qa, cache, self.c, positions=positions, q_to_seq=q_to_seq, slots=slots, block_table=md.block_table,
                               seq_lens=lens, scale=s.scale, window=s.window, gate=gate, sink=self.sink,
                               max_seq_len=md.max_seq_len or md.max_k)
        return ops.bmm_heads(lat, self.w_uv).reshape(T, s.heads * self.p)

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter, first row, rows, columns)}, columns None: a vector; or (store, shape)."""
        s, h, a = self.spec, self.hidden, self.in_proj.weight
        uq, kv, o = self._blocks()
        q_in = s.q_rank or h
        order = torch.arange(s.rot_dim)
        if s.rot_pairs:
            order = torch.cat([order[0::2], order[1::2]])

        def store_uq(w):
            w = w.view(s.heads, s.dim + s.rot_dim, q_in)
            uq[:, :s.dim, :q_in] = w[:, :s.dim]
            uq[:, self.d:self.d + s.rot_dim, :q_in] = w[:, s.dim:][:, order]

        def store_dkv(w):
            a.data[self.kv0:self.kv0 + s.kv_rank, :h] = w[:s.kv_rank]
            a.data[self.kv0 + s.kv_rank:self.kv0 + s.kv_rank + s.rot_dim, :h] = w[s.kv_rank:][order]

        def store_kv(row, n):
            def store(w):
                kv[:, row:row + n, :s.kv_rank] = w.view(s.heads, n, s.kv_rank)
            return store

        def store_o(w):
            o[:h, :, :s.vdim] = w.view(h, s.heads, s.vdim)

        t = {"dkv": (store_dkv, (s.kv_rank + s.rot_dim, h)), "dkv.norm": (self.kv_norm, 0, s.kv_rank, None),
             "uq" if s.q_rank else "q": (store_uq, (s.heads * (s.dim + s.rot_dim), q_in)),
             "uk": (store_kv(0, s.dim), (s.heads * s.dim, s.kv_rank)), "uv": (store_kv(self.d, s.vdim), (s.heads * s.vdim, s.kv_rank)),
             "o": (store_o, (h, s.heads * s.vdim))}
        if s.q_rank:
            t.update({"dq": (a, 0, s.q_rank, h), "dq.norm": (self.q_norm, 0, s.q_rank, None)})
        if s.gate:
            t["g"] = (a, self.g0, s.heads, h)
        if s.sink:
            t["sink"] = (self.sink, 0, s.heads, None)
        return t

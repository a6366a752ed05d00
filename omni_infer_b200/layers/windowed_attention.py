"""Softmax attention of the layer-list models: sliding window, optional RMSNorm over the whole q and the whole k projection,
rotation of the first dimensions of every head, key and value sizes of their own, optionally a sink per head in the softmax,
and optionally the cached keys and values of an earlier layer instead of own ones."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..models.config import AttentionSpec
from ..ops.layer_list import paged_attention, qk_norm_rope_cache
from .common import AttnMetadata, PaddedLinear


class WindowedAttention(nn.Module):
    def __init__(self, spec: AttentionSpec, hidden: int, eps: float, *, dtype, device=None, cos_sin=None, projections=True):
        """``projections=False``: a part of a larger mixer, which projects for it (rows q | k | v)."""
        super().__init__()
        self.spec, self.eps, self.cos_sin = spec, eps, cos_sin
        s = spec
        self.hkv = s.kv_heads if s.owns_kv else 0            # key/value heads this layer projects
        self.nq, self.nk, self.nv = s.heads * s.dim, self.hkv * s.dim, self.hkv * s.vdim
        self.proj_rows = self.nq + self.nk + self.nv
        if projections:
            self.qkv_proj = PaddedLinear(hidden, self.proj_rows, dtype=dtype, device=device)
            self.o_proj = PaddedLinear(s.heads * s.vdim, hidden, dtype=dtype, device=device)
        vec = lambda n: nn.Parameter(torch.ones(n, dtype=torch.float32, device=device), requires_grad=False)  # noqa: E731
        self.q_norm = vec(self.nq) if s.qk_norm else None
        self.k_norm = vec(self.nk) if s.qk_norm and self.hkv else None
        self.sink = nn.Parameter(torch.zeros(s.heads, dtype=torch.float32, device=device), requires_grad=False) if s.sink else None

    def forward(self, x, md: AttnMetadata, kv_cache):
        """``kv_cache``: (k, v) of the layer whose keys this one reads."""
        return ops.gemm(self.attend(ops.gemm(x, self.qkv_proj.weight), md, kv_cache), self.o_proj.weight)

    def attend(self, qkv, md: AttnMetadata, kv_cache, out=None, out_scale: float = 1.0):
        """Between the projections; ``out``: where the heads go (first columns), times ``out_scale``."""
        s = self.spec
        k_cache, v_cache = kv_cache
        qk_norm_rope_cache(qkv, s.heads, self.hkv, s.dim, s.vdim, self.q_norm, self.k_norm, self.eps, self.cos_sin, s.rot_dims,
                           md.positions, md.slot_mapping, k_cache, v_cache)
        q = qkv[:, :self.nq].unflatten(1, (s.heads, s.dim))
        ragged = md.is_prefill
        return paged_attention(q, k_cache, v_cache, positions=md.positions, q_to_seq=md.q_to_seq, slots=md.slot_mapping,
                               block_table=md.block_table, seq_lens=md.seq_lens if ragged else md.q_seq_lens, scale=s.scale,
                               window=s.window, cu_q=md.cu_q if ragged else None, max_q=md.max_q, max_seq_len=md.max_seq_len,
                               sink=self.sink, out_scale=out_scale, out=out)

    def input_targets(self, proj, h):
        """{checkpoint suffix: (parameter, first row, rows, columns)} of what comes before the output projection."""
        t = {"q": (proj, 0, self.nq, h)}
        if self.hkv:
            t.update({"k": (proj, self.nq, self.nk, h), "v": (proj, self.nq + self.nk, self.nv, h)})
        for name, p in (("q.norm", self.q_norm), ("k.norm", self.k_norm), ("sink", self.sink)):
            if p is not None:
                t[name] = (p, 0, p.shape[0], None)
        return t

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter, first row, rows, columns)}; columns None: a vector."""
        return dict(self.input_targets(self.qkv_proj.weight, self.qkv_proj.real_in),
                    o=(self.o_proj.weight, 0, self.o_proj.real_out, self.spec.heads * self.spec.vdim))

"""Softmax attention of the layer-list models: sliding window (optionally with kept first tokens) or chunks, optional RMSNorm over
the whole q and the whole k projection or over every head, rotation of the first dimensions of every head, key and value sizes of
their own, optionally a sink per head in the softmax, a soft cap of the scores, a distance bias, biases of the projections, a short
convolution of q, k and v, values mixed with an earlier layer's or divided by their root mean square, a learned logarithmic distance
bias, a sigmoid gate per element on the output, and the cached keys and values of an earlier layer instead of own ones."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..models.config import AttentionSpec
from ..ops.attn_prepare import qkv_prepare
from ..ops.layer_list import pad8, paged_attention, qk_norm_rope_cache, short_conv
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
        self.gate0 = pad8(self.proj_rows)                     # the gate's rows come after the others, from a multiple of 8 on
        self.n_out = s.heads * s.vdim
        if projections:
            self.qkv_proj = PaddedLinear(hidden, self.gate0 + self.n_out if s.out_gate else self.proj_rows, dtype=dtype, device=device, bias_column=s.bias)
            self.o_proj = PaddedLinear(s.heads * s.vdim, hidden, dtype=dtype, device=device)
        vec = lambda n: nn.Parameter(torch.ones(n, dtype=torch.float32, device=device), requires_grad=False)  # noqa: E731
        self.q_norm = vec(self.nq) if s.qk_norm else (vec(s.dim) if s.head_norm else None)
        self.k_norm = vec(self.nk) if s.qk_norm and self.hkv else (vec(s.dim) if s.head_norm else None)
        self.sink = nn.Parameter(torch.zeros(s.heads, dtype=torch.float32, device=device), requires_grad=False) if s.sink else None
        self.by_head = s.head_norm or s.rot_pairs or s.v_mix or s.v_norm or s.conv > 0
        if self.by_head and not self.hkv:
            raise ValueError("head norms, pairwise rotation, convolutions, mixed and normed values need keys and values of the layer's own")
        if s.out_gate and (s.conv or not projections):
            raise ValueError("an output gate needs the layer's own projections, without a convolution behind them")
        f32 = lambda *n: nn.Parameter(torch.zeros(*n, dtype=torch.float32, device=device), requires_grad=False)      # noqa: E731
        self.ones, self.out_bias = s.bias, f32(hidden) if s.bias else None       # the output's bias is added with the residual
        self.conv_weight = f32(s.conv, self.proj_rows) if s.conv else None       # taps first: channels are contiguous
        self.r1, self.r2 = (f32(s.heads), f32(s.heads)) if s.log_bias else (None, None)
        if s.log_bias:
            self.r1.init_value, self.r2.init_value = 0.5, 0.1
        self.vmix = f32(1) if s.v_mix else None
        if s.v_mix:
            self.vmix.init_value = 0.5
        slopes = 2.0 ** (-8.0 * torch.arange(1, s.heads + 1, dtype=torch.float64) / s.heads) if s.distance_bias else None
        self.register_buffer("slopes", slopes.float().to(device or "cpu") if slopes is not None else None, persistent=False)

    @property
    def in_cols(self):
        return self.qkv_proj.in_features

    def zero_padding(self):
        if self.spec.out_gate:
            self.qkv_proj.weight.data[self.proj_rows:self.gate0] = 0

    def state_shapes(self, slots: int, dtype):
        """Shapes and types of the state tensors for ``slots`` requests (layers with a convolution)."""
        return (((slots, self.spec.conv - 1, self.proj_rows), dtype),)

    def forward(self, x, md: AttnMetadata, kv_cache, shared=None):
        """``kv_cache``: (k, v) of the layer whose keys this one reads; with a convolution ((k, v), its state).  ``shared``: what the
        layers of one step hand on; the first layer that mixes its values leaves them there."""
        s = self.spec
        qkv = ops.gemm(x, self.qkv_proj.weight)
        if s.conv:
            kv_cache, (conv_state,) = kv_cache
            qkv = short_conv(qkv[:, :self.proj_rows], self.conv_weight, None, conv_state, positions=md.positions, state_slots=md.state_slots,
                             q_to_seq=md.q_to_seq, cu_q=md.cu_q if md.is_prefill else None)
        first = None
        if s.v_mix:
            first = shared.get("values")
            if first is None:
                shared["values"] = qkv[:, self.nq + self.nk:self.proj_rows]
        return ops.gemm(self.attend(qkv, md, kv_cache, first=first), self.o_proj.weight)

    def attend(self, qkv, md: AttnMetadata, kv_cache, out=None, out_scale: float = 1.0, first=None):
        """Between the projections; ``out``: where the heads go (first columns), times ``out_scale``.  ``first``: values to mix in."""
        s = self.spec
        k_cache, v_cache = kv_cache
        if self.by_head:
            qkv_prepare(qkv, s.heads, self.hkv, s.dim, s.vdim, self.q_norm, self.k_norm, self.eps, self.cos_sin, s.rot_dims, s.rot_pairs,
                        md.positions, md.slot_mapping, k_cache, v_cache, mix=self.vmix if first is not None else None, v_first=first,
                        v_norm=s.v_norm)
        else:
            qk_norm_rope_cache(qkv, s.heads, self.hkv, s.dim, s.vdim, self.q_norm, self.k_norm, self.eps, self.cos_sin, s.rot_dims,
                               md.positions, md.slot_mapping, k_cache, v_cache)
        q = qkv[:, :self.nq].unflatten(1, (s.heads, s.dim))
        ragged = md.is_prefill
        return paged_attention(q, k_cache, v_cache, positions=md.positions, q_to_seq=md.q_to_seq, slots=md.slot_mapping,
                               block_table=md.block_table, seq_lens=md.seq_lens if ragged else md.q_seq_lens, scale=s.scale,
                               window=s.window, cu_q=md.cu_q if ragged else None, max_q=md.max_q, max_seq_len=md.max_seq_len,
                               sink=self.sink, out_scale=out_scale, out=out, keep_first=s.keep_first, chunk=s.chunk,
                               softcap=s.softcap, slopes=self.slopes, log_bias=(self.r1, self.r2) if s.log_bias else None,
                               gate=qkv[:, self.gate0:self.gate0 + self.n_out] if s.out_gate else None)

    def input_targets(self, proj, h):
        """{checkpoint suffix: (parameter, first row, rows, columns)} of what comes before the output projection."""
        t = {"q": (proj, 0, self.nq, h)}
        if self.hkv:
            t.update({"k": (proj, self.nq, self.nk, h), "v": (proj, self.nq + self.nk, self.nv, h)})
        for name, p in (("q.norm", self.q_norm), ("k.norm", self.k_norm), ("sink", self.sink), ("vmix", self.vmix),
                        ("r1", self.r1), ("r2", self.r2)):
            if p is not None:
                t[name] = (p, 0, p.shape[0], None)
        return t

    def _parts(self):
        return ("q", 0, self.nq), ("k", self.nq, self.nk), ("v", self.nq + self.nk, self.nv)

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter, first row, rows, columns)}; columns None: a vector."""
        s = self.spec
        t = dict(self.input_targets(self.qkv_proj.weight, self.qkv_proj.real_in),
                 o=(self.o_proj.weight, 0, self.o_proj.real_out, s.heads * s.vdim))
        if s.out_gate:
            t["g"] = (self.qkv_proj.weight, self.gate0, self.n_out, self.qkv_proj.real_in)
        if s.bias:
            t.update({c + ".b": self.qkv_proj.bias_target(a, n) for c, a, n in self._parts()})
            t["o.b"] = (self.out_bias, 0, self.o_proj.real_out, None)
        if s.conv:      # stored transposed
            t.update({c + ".conv": (self.conv_weight.data[:, a:a + n], 0, s.conv, -n) for c, a, n in self._parts()})
        return t

"""Mixers with a matrix per head as their state: WKV time mixing, gated linear attention, and attention beside the matrix memory
of xLSTM.
A request's state lives in its state slot, the attention's keys and values in its pages."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..models.config import GLASpec, MLSTMSpec, ParallelSpec, WkvSpec
from ..ops.layer_list import pad8
from ..ops.matrix_state import CHUNK_MIN_ROWS, gla_scan, head_norm, mlstm_chunked, mlstm_gates, mlstm_scan, wkv_scan
from ..ops.streams import tanh_split, token_shift
from .common import AttnMetadata, PaddedLinear
from .windowed_attention import WindowedAttention


def _f32(*n, device=None, value=None):
    p = nn.Parameter(torch.full(n, value if value is not None else 0.0, dtype=torch.float32, device=device), requires_grad=False)
    p.init_value = value
    return p


def _pad64(n: int) -> int:
    return (n + 63) // 64 * 64


def _ragged(md: AttnMetadata) -> dict:
    """Arguments that tell an op which rows belong to which request."""
    return dict(positions=md.positions, state_slots=md.state_slots, cu_q=md.cu_q if md.is_prefill else None)


def _rows_of(md: AttnMetadata) -> dict:
    return dict(min_q=min(md.query_lens) if md.is_prefill else 1, max_q=md.max_q)


class MLSTM(nn.Module):
    """Matrix memory between its projections.  Its rows of the input projection: q | k | v | output gate, each block starting at
    a multiple of 8."""

    def __init__(self, spec: MLSTMSpec, eps: float, device=None):
        super().__init__()
        self.spec, self.eps = spec, eps
        s = spec
        self.nk, self.nv = s.heads * s.dim, s.heads * s.vdim
        self.k0 = pad8(self.nk)
        self.v0 = 2 * self.k0
        self.g0 = self.v0 + pad8(self.nv)
        self.proj_rows = self.g0 + pad8(self.nv)
        self.f_col = pad8(s.heads)                     # of the forget gates in the gate projection
        self.i_bias, self.f_bias = _f32(s.heads, device=device), _f32(s.heads, device=device, value=3.0)
        self.norm_weight = nn.Parameter(torch.ones(self.nv, dtype=torch.float32, device=device), requires_grad=False)

    def state_shapes(self, slots: int, dtype):
        s = self.spec
        return (((slots, s.heads, s.vdim + 1, s.dim), torch.float32), ((slots, s.heads), torch.float32))

    def mix(self, u, z, md: AttnMetadata, state, out, scale):
        """u: this mixer's part of the projected rows, z: gates before their biases (fp32).  Writes scale * (o W_norm gate)."""
        s, where = self.spec, _ragged(md)
        S, m = state
        chunks = u.is_cuda and md.is_prefill and mlstm_chunked(u.dtype, s.dim, s.vdim) and md.max_q >= CHUNK_MIN_ROWS
        gates = mlstm_gates(z, self.f_col, self.i_bias, self.f_bias, s.gate_cap, m, chunks=chunks, **where)
        y = mlstm_scan(u[:, :self.nk], u[:, self.k0:self.k0 + self.nk], u[:, self.v0:self.v0 + self.nv], gates, S, H=s.heads,
                       P=s.vdim, N=s.dim, **where, **_rows_of(md))
        return head_norm(y, u[:, self.g0:], self.norm_weight, out, H=s.heads, P=s.vdim, eps=self.eps, act="sigmoid", scale=scale,
                         gates=gates)

    def checkpoint_targets(self, proj, row0, gate_proj, h):
        return {"q": (proj, row0, self.nk, h), "k": (proj, row0 + self.k0, self.nk, h), "v": (proj, row0 + self.v0, self.nv, h),
                "g": (proj, row0 + self.g0, self.nv, h), "i": (gate_proj, 0, self.spec.heads, h),
                "f": (gate_proj, self.f_col, self.spec.heads, h), "i.b": (self.i_bias, 0, self.spec.heads, None),
                "f.b": (self.f_bias, 0, self.spec.heads, None), "norm": (self.norm_weight, 0, self.nv, None)}


class ParallelMixer(nn.Module):
    """left_scale * attention + right_scale * matrix memory on the same input: one input projection for both, one fp32 projection
    for the gates, and one output projection over both (the scales enter before its input is rounded)."""

    def __init__(self, spec: ParallelSpec, hidden: int, eps: float, *, dtype, device=None, cos_sin=None):
        super().__init__()
        self.spec, self.hidden = spec, hidden
        self.left = WindowedAttention(spec.left, hidden, eps, dtype=dtype, device=device, cos_sin=cos_sin, projections=False)
        self.right = MLSTM(spec.right, eps, device)
        self.right0 = pad8(self.left.proj_rows)        # first row of the matrix memory in the input projection
        self.n_left = spec.left.heads * spec.left.vdim
        self.o_right0 = pad8(self.n_left)
        self.in_proj = PaddedLinear(hidden, self.right0 + self.right.proj_rows, dtype=dtype, device=device)
        self.gate_proj = PaddedLinear(hidden, 2 * self.right.f_col, dtype=dtype, device=device)
        self.o_proj = PaddedLinear(self.o_right0 + self.right.nv, hidden, dtype=dtype, device=device)

    def zero_padding(self):
        w, o, r = self.in_proj.weight.data, self.o_proj.weight.data, self.right
        w[self.left.proj_rows:self.right0] = 0
        for a, n in ((0, r.nk), (r.k0, r.nk), (r.v0, r.nv), (r.g0, r.nv)):
            w[self.right0 + a + n:self.right0 + a + pad8(n)] = 0
        self.gate_proj.weight.data[r.spec.heads:r.f_col] = 0
        self.gate_proj.weight.data[r.f_col + r.spec.heads:] = 0
        o[:, self.n_left:self.o_right0] = 0

    def state_shapes(self, slots: int, dtype):
        return self.right.state_shapes(slots, dtype)

    def forward(self, x, md: AttnMetadata, cache):
        """``cache``: (pages of the attention, state slots of the matrix memory)."""
        pages, state = cache
        u = ops.gemm(x, self.in_proj.weight)
        z = ops.gemm(x, self.gate_proj.weight, out_dtype=torch.float32)
        K = self.o_proj.in_features
        full = self.n_left == self.o_right0 and K == self.o_proj.real_in
        both = (torch.empty if full else torch.zeros)(x.shape[0], K, dtype=x.dtype, device=x.device)
        self.left.attend(u, md, pages, out=both, out_scale=self.spec.left_scale)
        self.right.mix(u[:, self.right0:], z, md, state, both[:, self.o_right0:], self.spec.right_scale)
        return ops.gemm(both, self.o_proj.weight)

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter or a view of one, first row, rows, columns)}; columns None: a vector."""
        w, h, o = self.in_proj.weight, self.hidden, self.o_proj.weight
        t = {"left." + k: v for k, v in self.left.input_targets(w, h).items()}
        t["left.o"] = (o, 0, h, self.n_left)
        t.update({"right." + k: v for k, v in self.right.checkpoint_targets(w, self.right0, self.gate_proj.weight, h).items()})
        t["right.o"] = (o.data[:, self.o_right0:], 0, h, self.right.nv)
        return t


class WkvMixer(nn.Module):
    """WKV time mixing.  The shifted inputs of r, k, v and the gate lie side by side, so their projections are one grouped GEMM;
    the decay goes through a low-rank projection whose values stay fp32 (the tanh between as bf16 hi | lo)."""

    def __init__(self, spec: WkvSpec, hidden: int, eps: float, *, dtype, device=None):
        super().__init__()
        self.spec, self.hidden, self.eps = spec, hidden, eps
        s = spec
        if s.rank < 1:
            raise ValueError("the rank of the decay's projection is not known: it is the number of rows of mix.w1")
        self.inner, self.part = s.heads * s.dim, _pad64(hidden)
        self.block, self.half = pad8(self.inner), pad8(s.rank)
        w = lambda *n: nn.Parameter(torch.zeros(*n, dtype=dtype, device=device), requires_grad=False)  # noqa: E731
        self.rkvg = w(4, self.block, self.part)
        self.w1 = w(self.half, self.part)
        self.w2 = w(self.block, self.half if dtype == torch.float32 else 2 * self.half)      # twice side by side in bf16
        self.o_proj = PaddedLinear(self.inner, hidden, dtype=dtype, device=device)
        self.mu = _f32(5, hidden, device=device, value=0.5)                  # r, k, v, g, w
        self.w0, self.u = _f32(self.inner, device=device, value=-1.0), _f32(self.inner, device=device, value=0.3)
        self.norm_weight = nn.Parameter(torch.ones(self.inner, dtype=torch.float32, device=device), requires_grad=False)

    def zero_padding(self):
        self.rkvg.data[:, self.inner:] = 0
        self.rkvg.data[:, :, self.hidden:] = 0
        self.w1.data[self.spec.rank:] = 0
        self.w1.data[:, self.hidden:] = 0
        self.w2.data[self.inner:] = 0
        self.w2.data[:, self.spec.rank:self.half] = 0
        if self.w2.shape[1] > self.half:
            self.w2.data[:, self.half:] = self.w2.data[:, :self.half]

    def state_shapes(self, slots: int, dtype):
        s = self.spec
        return (((slots, self.hidden), dtype), ((slots, s.heads, s.dim, s.dim), torch.float32))

    def forward(self, x, md: AttnMetadata, state):
        s, where, n = self.spec, _ragged(md), self.inner
        last, S = state
        xs = token_shift(x, self.mu, last, self.part, q_to_seq=md.q_to_seq, **where)
        p = ops.bmm_heads(xs[:, :4], self.rkvg)
        a = ops.gemm(xs[:, 4], self.w1, out_dtype=torch.float32)
        z = ops.gemm(tanh_split(a, s.rank, x.dtype), self.w2, out_dtype=torch.float32)
        y = wkv_scan(p[:, 0, :n], p[:, 1, :n], p[:, 2, :n], z, self.w0, self.u, S, H=s.heads, N=s.dim, **where, **_rows_of(md))
        out = (torch.empty if self.o_proj.in_features == n else torch.zeros)(x.shape[0], self.o_proj.in_features, dtype=x.dtype,
                                                                            device=x.device)
        head_norm(y, p[:, 3], self.norm_weight, out, H=s.heads, P=s.dim, eps=self.eps, act="silu")
        return ops.gemm(out, self.o_proj.weight)

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter or a view of one, first row, rows, columns)}; columns None: a vector."""
        s, h, n = self.spec, self.hidden, self.inner
        t = {c: (self.rkvg.data[i], 0, n, h) for i, c in enumerate("rkvg")}
        t.update({"mu." + c: (self.mu.data[i], 0, h, None) for i, c in enumerate("rkvgw")})
        t.update({"w1": (self.w1, 0, s.rank, h), "w2": (self.w2, 0, n, s.rank), "w0": (self.w0, 0, n, None),
                  "u": (self.u.data.view(s.heads, s.dim), 0, s.heads, s.dim), "norm": (self.norm_weight, 0, n, None),
                  "o": (self.o_proj.weight, 0, h, n)})
        return t


class GlaMixer(nn.Module):
    """Gated linear attention.  One input projection with rows q | k | v | output gate | first half of the decay's projection, each
    block from a multiple of 8 on; the second half's values stay fp32."""
    out_bias = None
    ones = False

    def __init__(self, spec: GLASpec, hidden: int, eps: float, *, dtype, device=None):
        super().__init__()
        self.spec, self.hidden, self.eps = spec, hidden, eps
        s = spec
        if s.rank < 1:
            raise ValueError("the rank of the decay's projection is not known: it is the number of rows of mix.a1")
        self.nk, self.nv, self.half = s.heads * s.dim, s.heads * s.vdim, pad8(s.rank)
        self.k0 = pad8(self.nk)
        self.v0 = 2 * self.k0
        self.g0 = self.v0 + pad8(self.nv)
        self.a0 = self.g0 + pad8(self.nv)
        self.in_proj = PaddedLinear(hidden, self.a0 + self.half, dtype=dtype, device=device)
        self.a2 = nn.Parameter(torch.zeros(self.k0, self.half, dtype=dtype, device=device), requires_grad=False)
        self.o_proj = PaddedLinear(self.nv, hidden, dtype=dtype, device=device)
        self.decay_bias = _f32(self.nk, device=device, value=2.0)
        self.norm_weight = nn.Parameter(torch.ones(self.nv, dtype=torch.float32, device=device), requires_grad=False)      # of every head

    @property
    def in_cols(self):
        return self.in_proj.in_features

    def _parts(self):
        return (("q", 0, self.nk), ("k", self.k0, self.nk), ("v", self.v0, self.nv), ("g", self.g0, self.nv), ("a1", self.a0, self.spec.rank))

    def zero_padding(self):
        w = self.in_proj.weight.data
        for _, a, n in self._parts():
            w[a + n:a + pad8(n)] = 0
        self.a2.data[self.nk:] = 0
        self.a2.data[:, self.spec.rank:] = 0

    def state_shapes(self, slots: int, dtype):
        s = self.spec
        return (((slots, s.heads, s.vdim, s.dim), torch.float32),)

    def forward(self, x, md: AttnMetadata, state, shared=None):
        s, nk = self.spec, self.nk
        u = ops.gemm(x, self.in_proj.weight)
        z = ops.gemm(u[:, self.a0:], self.a2, out_dtype=torch.float32)
        y = gla_scan(u[:, :nk], u[:, self.k0:self.k0 + nk], u[:, self.v0:self.v0 + self.nv], z, self.decay_bias, 1.0 / s.tau, state[0],
                     H=s.heads, P=s.vdim, N=s.dim, **_ragged(md), **_rows_of(md))
        K = self.o_proj.in_features
        out = (torch.empty if K == self.nv else torch.zeros)(x.shape[0], K, dtype=x.dtype, device=x.device)
        head_norm(y, u[:, self.g0:self.a0], self.norm_weight, out, H=s.heads, P=s.vdim, eps=self.eps, act="silu")
        return ops.gemm(out, self.o_proj.weight)

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter or a view of one, first row, rows, columns)}; columns None: a vector; or (store, shape)."""
        s, h, w = self.spec, self.hidden, self.in_proj.weight

        def store_norm(v):
            self.norm_weight.data.view(s.heads, s.vdim).copy_(v.float())

        t = {name: (w, a, n, h) for name, a, n in self._parts()}
        t.update({"a2": (self.a2, 0, self.nk, s.rank), "a2.b": (self.decay_bias, 0, self.nk, None), "norm": (store_norm, (s.vdim,)),
                  "o": (self.o_proj.weight, 0, h, self.nv)})
        return t

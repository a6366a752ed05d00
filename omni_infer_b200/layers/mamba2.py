"""Mamba-2 mixer: input projection, short causal convolution, state-space recurrence, gate, grouped norm, output
projection.  A request's convolution inputs and fp32 state live in its state slot."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..models.config import Mamba2Spec
from ..ops.layer_list import conv_silu, gated_group_norm, ssm_scan
from .common import AttnMetadata, PaddedLinear


class Mamba2Mixer(nn.Module):
    def __init__(self, spec: Mamba2Spec, hidden: int, eps: float, *, dtype, device=None):
        super().__init__()
        self.spec, self.eps = spec, eps
        s = spec
        # rows: z | x | B | C | dt
        self.in_proj = PaddedLinear(hidden, s.inner + s.conv_channels + s.heads, dtype=dtype, device=device)
        self.o_proj = PaddedLinear(s.inner, hidden, dtype=dtype, device=device)
        f32 = lambda *n: nn.Parameter(torch.zeros(*n, dtype=torch.float32, device=device), requires_grad=False)  # noqa: E731
        self.conv_weight = f32(s.conv, s.conv_channels)      # taps first: channels are contiguous
        self.conv_bias, self.dt_bias, self.A_log, self.D = f32(s.conv_channels), f32(s.heads), f32(s.heads), f32(s.heads)
        self.norm_weight = nn.Parameter(torch.ones(s.inner, dtype=torch.float32, device=device), requires_grad=False)

    def state_shapes(self, slots: int, dtype):
        """Shapes and types of the state tensors for ``slots`` requests."""
        s = self.spec
        return (((slots, s.conv - 1, s.conv_channels), dtype), ((slots, s.heads, s.vdim, s.state), torch.float32))

    def forward(self, x, md: AttnMetadata, state):
        s = self.spec
        conv_state, ssm_state = state
        u = ops.gemm(x, self.in_proj.weight)
        cu_q = md.cu_q if md.is_prefill else None
        xbc = conv_silu(u[:, s.inner:s.inner + s.conv_channels], self.conv_weight, self.conv_bias, conv_state,
                        positions=md.positions, state_slots=md.state_slots, q_to_seq=md.q_to_seq, cu_q=cu_q)
        dt = u[:, s.inner + s.conv_channels:s.inner + s.conv_channels + s.heads]
        y = ssm_scan(xbc, dt, self.A_log, self.dt_bias, self.D, ssm_state, H=s.heads, P=s.vdim,
                     N=s.state, G=s.groups, positions=md.positions, state_slots=md.state_slots, cu_q=cu_q,
                     min_q=min(md.query_lens) if md.is_prefill else 1, max_q=md.max_q)
        return ops.gemm(gated_group_norm(y, u, self.norm_weight, s.norm_groups, self.eps), self.o_proj.weight)

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter, first row, rows, columns)}; columns None: a vector, negative: stored transposed."""
        s = self.spec
        return {"in": (self.in_proj.weight, 0, self.in_proj.real_out, self.in_proj.real_in),
                "conv": (self.conv_weight, 0, s.conv, -s.conv_channels), "conv.b": (self.conv_bias, 0, s.conv_channels, None),
                "dt_bias": (self.dt_bias, 0, s.heads, None), "A_log": (self.A_log, 0, s.heads, None), "D": (self.D, 0, s.heads, None),
                "norm": (self.norm_weight, 0, s.inner, None),
                "o": (self.o_proj.weight, 0, self.o_proj.real_out, s.inner)}

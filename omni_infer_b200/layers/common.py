"""Building blocks shared by every model: attention metadata, linear layers (bf16 / block-scaled
e4m3), RMSNorm, the SwiGLU MLP."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..ops import FP8


@dataclass
class AttnMetadata:
    """Per-step attention inputs built by the model runner.

    The reference carries the same information in AscendMLAMetadata / AscendMetadata
    (omni/models/common/layers/attention/backend/mla.py:105-166): attention state, slot mapping,
    block table, sequence lengths; prefill additionally has ragged query/key offsets."""
    is_prefill: bool
    positions: torch.Tensor                 # [T] int64
    slot_mapping: torch.Tensor              # [T] int64, -1 = do not store
    block_table: torch.Tensor               # [B, max_blocks] int32
    seq_lens: torch.Tensor                  # [B] int32 total kv tokens per request after this step
    # prefill
    cu_q: Optional[torch.Tensor] = None     # [B+1] int32
    cu_k: Optional[torch.Tensor] = None     # [B+1] int32
    query_lens: Optional[list] = None
    context_lens: Optional[list] = None     # cached-prefix tokens per request
    max_q: int = 0
    max_k: int = 0
    kv_gather_slots: Optional[torch.Tensor] = None   # [sum_k] int64 cache slots of the whole context (prefix hits)
    # decode
    tokens_per_req: int = 1                 # 1 + speculative tokens
    q_seq_lens: Optional[torch.Tensor] = None   # [B * tokens_per_req] int32 visible kv tokens per q row
    q_to_seq: Optional[torch.Tensor] = None     # [B * tokens_per_req] int32 (prefill: [T], the request of every row)
    max_seq_len: int = 0
    num_valid: Optional[torch.Tensor] = None    # device int32 scalar: rows beyond are padding
    sample_indices: Optional[torch.Tensor] = None  # rows of hidden states that produce logits
    state_slots: Optional[torch.Tensor] = None     # [B] int32 recurrent-state slot per request, -1 = padding row
    # Omni-Attention (compressed layers): per-layer-group overrides
    omni: Optional[dict] = None
    plans: dict = field(default_factory=dict)      # what layers have worked out for this step and share


def _dtype(name: str) -> torch.dtype:
    return {"float32": torch.float32, "bfloat16": torch.bfloat16, "float16": torch.float16}[name]


class Linear(nn.Module):
    """y = x W^T (+ b).  ``quant='fp8_block'`` stores e4m3 weights with 128x128 scales and quantises the
    activation per (row, 128 columns) unless the caller passes it already quantised."""

    def __init__(self, in_features: int, out_features: int, *, dtype=torch.bfloat16, quant: str = "none",
                 bias: bool = False, device=None):
        super().__init__()
        self.in_features, self.out_features, self.quant = in_features, out_features, quant
        if quant == "fp8_block":
            self.weight = nn.Parameter(torch.empty(out_features, in_features, dtype=FP8, device=device),
                                       requires_grad=False)
            self.weight_scale = nn.Parameter(
                torch.ones((out_features + 127) // 128, (in_features + 127) // 128, dtype=torch.float32, device=device),
                requires_grad=False)
        else:
            self.weight = nn.Parameter(torch.empty(out_features, in_features, dtype=dtype, device=device),
                                       requires_grad=False)
            self.weight_scale = None
        self.bias = nn.Parameter(torch.zeros(out_features, dtype=dtype, device=device), requires_grad=False) if bias else None

    def forward(self, x, xq=None, epi: str = "store", out_dtype=None):
        if self.quant == "fp8_block":
            if xq is None:
                xq = ops.quant_fp8_block(x)
            y = ops.gemm(xq[0], self.weight, w_scale=self.weight_scale, x_scale=xq[1], epi=epi, out_dtype=out_dtype)
        else:
            y = ops.gemm(x, self.weight, epi=epi, out_dtype=out_dtype)
        if self.bias is not None:
            y = y + self.bias
        return y


class RMSNorm(nn.Module):
    def __init__(self, hidden: int, eps: float, dtype=torch.bfloat16, device=None):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(hidden, dtype=dtype, device=device), requires_grad=False)
        self.eps = eps

    def forward(self, x, residual=None, quant=False):
        """Returns y, or (y, y_q, scale) with ``quant``; ``residual`` is updated in place to x + residual."""
        return ops.rmsnorm(x, self.weight, self.eps, residual=residual, quant=quant)


class PaddedLinear(Linear):
    """Linear whose stored weight has both sizes rounded up to a multiple of 8 (TMA row pitch, 16-byte output vectors).  The
    padding is zero and activations carry zeros in their padding columns, so the product is that of the real sizes."""

    def __init__(self, in_features: int, out_features: int, *, dtype=torch.bfloat16, device=None, bias_column: bool = False):
        """``bias_column``: one more column holds the biases; activations carry a one there (``ops.layer_list.add_norm``)."""
        self.bias_column = bias_column
        # with the extra column the rows would start at odd 16-byte steps: whole 128-byte lines keep the product as fast as without it
        align = 64 if bias_column else 8
        super().__init__((in_features + int(bias_column) + align - 1) // align * align, (out_features + 7) // 8 * 8, dtype=dtype, device=device)
        self.real_in, self.real_out = in_features, out_features
        self.zero_padding()

    def zero_padding(self):
        self.weight.data[self.real_out:] = 0
        self.weight.data[:, self.real_in + int(self.bias_column):] = 0

    def bias_target(self, row0: int, rows: int):
        """Checkpoint target of the biases of those rows."""
        return self.weight.data[:, self.real_in], row0, rows, None


class GeGLUMLP(nn.Module):
    """gate_up (merged, gate rows first, each block padded to a multiple of 8) -> gelu (tanh form) of the gate times up,
    in the GEMM epilogue where the width allows -> down.  ``epi="swiglu"``: silu of the gate.  ``bias``: all three projections
    have one; the last is left to the caller, who adds it with the residual."""
    epi = "geglu"

    def __init__(self, hidden: int, inter: int, *, dtype=torch.bfloat16, device=None, epi=None, bias: bool = False):
        super().__init__()
        self.epi = epi or self.epi
        self.inter, self.block, self.limit, self.ones = inter, (inter + 7) // 8 * 8, 0.0, bias
        self.gate_up_proj = PaddedLinear(hidden, 2 * self.block, dtype=dtype, device=device, bias_column=bias)
        self.down_proj = PaddedLinear(inter, hidden, dtype=dtype, device=device)
        self.out_bias = nn.Parameter(torch.zeros(hidden, dtype=torch.float32, device=device), requires_grad=False) if bias else None
        self.zero_padding()

    @property
    def in_cols(self):
        return self.gate_up_proj.in_features

    def zero_padding(self):
        w = self.gate_up_proj.weight.data
        w[self.inter:self.block] = 0
        w[self.block + self.inter:] = 0

    def forward(self, x):
        return ops.gemm(ops.gemm(x, self.gate_up_proj.weight, epi=self.epi, glu_limit=self.limit), self.down_proj.weight)

    def checkpoint_targets(self):
        """{checkpoint suffix: (parameter, first row, rows, columns)}."""
        w, h = self.gate_up_proj.weight, self.gate_up_proj.real_in
        t = {"gate": (w, 0, self.inter, h), "up": (w, self.block, self.inter, h), "down": (self.down_proj.weight, 0, h, self.inter)}
        if self.out_bias is not None:
            t.update({"gate.b": self.gate_up_proj.bias_target(0, self.inter), "up.b": self.gate_up_proj.bias_target(self.block, self.inter),
                      "down.b": (self.out_bias, 0, h, None)})
        return t


class ClampedGLUMLP(GeGLUMLP):
    """The same with g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(1.702 g) (u + 1)."""
    epi = "clamped_glu"

    def __init__(self, hidden: int, inter: int, limit: float, *, dtype=torch.bfloat16, device=None):
        super().__init__(hidden, inter, dtype=dtype, device=device)
        self.limit = limit


class PostNorm(nn.Module):
    """Norm on a sublayer's output: residual (fp32, in place) += rmsnorm(y) * weight, in one kernel with the activation copy
    that the next sublayer reads.  The weight is kept in fp32."""

    def __init__(self, hidden: int, eps: float, device=None):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(hidden, dtype=torch.float32, device=device), requires_grad=False)
        self.eps = eps

    def forward(self, y, residual):
        return ops.layer_list.post_norm_add(y, self.weight, residual, self.eps)


class SwiGLUMLP(nn.Module):
    """gate_up (merged, gate rows first) -> SwiGLU fused in the GEMM epilogue -> down."""

    def __init__(self, hidden: int, inter: int, *, dtype=torch.bfloat16, quant="none", device=None):
        super().__init__()
        self.gate_up_proj = Linear(hidden, 2 * inter, dtype=dtype, quant=quant, device=device)
        self.down_proj = Linear(inter, hidden, dtype=dtype, quant=quant, device=device)
        self.quant = quant

    def forward(self, x, xq=None):
        if self.quant == "fp8_block":
            if xq is None:
                xq = ops.quant_fp8_block(x)
            aq = ops.gemm(xq[0], self.gate_up_proj.weight, w_scale=self.gate_up_proj.weight_scale, x_scale=xq[1],
                          epi="swiglu_quant")
            return ops.gemm(aq[0], self.down_proj.weight, w_scale=self.down_proj.weight_scale, x_scale=aq[1])
        act = ops.gemm(x, self.gate_up_proj.weight, epi="swiglu")
        return ops.gemm(act, self.down_proj.weight)

"""Ops of models with several residual streams (hyper-connections) and layer norms ahead of the sublayers.

Streams are fp32 [T, streams, ld]; CUDA tensors run ``csrc/kernels/stream_ops.cu``, CPU tensors the fp32 references here."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _native as nat
from .layer_list import _f32, _segments, pad8


@dataclass
class ExpertSum:
    """Output of an expert mixture before its parts are added up: row ``row_of[t, k]`` of ``y`` (-1: none) for every choice of
    a token, the weights of its choices beyond ``experts`` times the sublayer's input, and the shared expert's rows."""
    y: torch.Tensor                    # [rows, ld], already weighted
    row_of: torch.Tensor               # int32 [T * k]
    ids: torch.Tensor                  # int32 [T, k]
    weights: torch.Tensor              # fp32 [T, k]
    experts: int
    h: torch.Tensor                    # [T, ld] the sublayer's input
    shared: Optional[torch.Tensor]     # [T, ld]

    def total(self) -> torch.Tensor:
        """fp32 [T, ld], in plain torch."""
        T, k = self.ids.shape
        rows = self.row_of.view(T, k).long()
        out = (self.y[rows.clamp_min(0)].float() * (rows >= 0).unsqueeze(-1)).sum(1)
        out = out + (self.weights * (self.ids >= self.experts)).sum(1, keepdim=True) * self.h.float()
        return out if self.shared is None else out + self.shared.float()


def layer_norm_ref(u, w, eps):
    c = u - u.mean(-1, keepdim=True)
    return c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * w


def _normed_ref(x, inw, w, eps, dtype):
    H = w.shape[0]
    h = torch.zeros(x.shape[0], x.shape[2], dtype=dtype)
    h[:, :H] = layer_norm_ref(torch.einsum("tsw,s->tw", x[:, :, :H], inw), w, eps).to(dtype)
    return h


def embed_streams(ids, table, width, scale, inw, w, eps):
    """Embedding rows times ``scale`` into every stream -> (streams, normed input of the first sublayer)."""
    T, ld, n = ids.shape[0], table.shape[1], inw.shape[0]
    if not table.is_cuda:
        x = (table[ids].float() * scale)[:, None].repeat(1, n, 1)
        return x, _normed_ref(x, inw, w, eps, table.dtype)
    x = (torch.empty if ld == width else torch.zeros)(T, n, ld, dtype=torch.float32, device=table.device)
    h = torch.empty(T, ld, dtype=table.dtype, device=table.device)
    rc = nat.lib().omni_embed_streams(nat.ptr(ids), nat.ptr(table), nat.c_int(table.shape[0]), nat.c_int(T), nat.c_int(width),
                                      nat.c_int(ld), nat.c_float(scale), nat.c_int(n), nat.ptr(inw), nat.ptr(w), nat.c_float(eps),
                                      nat.ptr(x), nat.ptr(h), nat.c_int(_f32(table)), nat.stream())
    nat.check_rc(rc, "omni_embed_streams")
    return x, h


def stream_step(x, y, mix, out, inw, w, eps, dtype, last=False):
    """x[:, t] <- sum_s mix[s, t] x[:, s] + out[t] y in place (left as it was with ``last`` on a GPU), returns the next sublayer's
    input layer_norm(sum_s inw[s] x[:, s]) w as activations of ``dtype``.  ``y``: rows, or an :class:`ExpertSum`."""
    T, n, ld = x.shape
    H = w.shape[0]
    es = y if isinstance(y, ExpertSum) else None
    if not x.is_cuda:
        yf = es.total() if es is not None else y.float()
        x[:, :, :H] = torch.einsum("tsw,sq->tqw", x[:, :, :H], mix) + out[None, :, None] * yf[:, None, :H]
        return _normed_ref(x, inw, w, eps, dtype)
    rows = es.y if es is not None else y
    assert rows.dtype == dtype and rows.stride(1) == 1
    if es is not None:
        assert es.h.is_contiguous() and es.h.shape[1] == ld and (es.shared is None or es.shared.stride(0) == rows.stride(0))
    h = torch.empty(T, ld, dtype=dtype, device=x.device)
    rc = nat.lib().omni_stream_step(
        nat.ptr(x), nat.c_int(T), nat.c_int(H), nat.c_int(ld), nat.c_int(n), nat.ptr(rows), nat.c_int(rows.stride(0)),
        nat.ptr(es.row_of if es else None), nat.ptr(es.ids if es else None), nat.ptr(es.weights if es else None),
        nat.c_int(es.ids.shape[1] if es else 0), nat.c_int(es.experts if es else 0), nat.ptr(es.h if es else None),
        nat.ptr(es.shared if es else None), nat.ptr(mix), nat.ptr(out), nat.ptr(inw), nat.ptr(w), nat.c_float(eps), nat.ptr(h),
        nat.c_int(ld), nat.c_int(int(last)), nat.c_int(_f32(h)), nat.stream())
    nat.check_rc(rc, "omni_stream_step")
    return h


# ----------------------------------------------------------------------------- token shift
def token_shift(h, mu, state, part_ld, *, positions, state_slots, q_to_seq=None, cu_q=None):
    """h + (h of the previous token - h) mu[k] for every row of ``mu`` [parts, H] -> [T, parts, part_ld] (zeros past H).
    ``state`` [slots, H] holds the last h of every request and is moved on; before a sequence's first token lie zeros."""
    T, (parts, H) = h.shape[0], mu.shape
    if not h.is_cuda:
        out = torch.zeros(T, parts, part_ld, dtype=h.dtype)
        for r, a, b in _segments(cu_q, T):
            slot = int(state_slots[r])
            first = state[slot].float() if slot >= 0 and int(positions[a]) > 0 else torch.zeros(H)
            x = h[a:b, :H].float()
            prev = torch.cat([first[None], x[:-1]])
            out[a:b, :, :H] = (x[:, None] + (prev - x)[:, None] * mu[None]).to(h.dtype)
            if slot >= 0:
                state[slot] = h[b - 1, :H]
        return out
    assert h.stride(1) == 1 and mu.is_contiguous() and state.dtype == h.dtype and state.is_contiguous()
    out = torch.empty(T, parts, part_ld, dtype=h.dtype, device=h.device)
    rc = nat.lib().omni_token_shift(
        nat.ptr(h), nat.c_int(h.stride(0)), nat.ptr(mu), nat.c_int(parts), nat.c_int(H), nat.ptr(state), nat.ptr(positions),
        nat.ptr(q_to_seq), nat.ptr(cu_q), nat.ptr(state_slots), nat.c_int(T), nat.ptr(out), nat.c_int(part_ld), nat.c_int(_f32(h)),
        nat.stream())
    nat.check_rc(rc, "omni_token_shift")
    return out


def tanh_split(a, rank, dtype):
    """tanh of fp32 [T, >= rank]: bf16 activations get [T, 2 pad8(rank)] = hi | lo with hi + lo = tanh to 16 bits, fp32 ones
    [T, pad8(rank)]; zeros past the rank."""
    T, half, f32 = a.shape[0], pad8(rank), dtype == torch.float32
    if not a.is_cuda:
        v = torch.zeros(T, half)
        v[:, :rank] = torch.tanh(a[:, :rank].float())
        hi = v.to(dtype)
        return hi if f32 else torch.cat([hi, (v - hi.float()).to(dtype)], 1)
    assert a.dtype == torch.float32 and a.stride(1) == 1
    out = torch.empty(T, half if f32 else 2 * half, dtype=dtype, device=a.device)
    rc = nat.lib().omni_tanh_split(nat.ptr(a), nat.c_int(a.stride(0)), nat.c_int(rank), nat.ptr(out), nat.c_int(half), nat.c_int(T),
                                   nat.c_int(int(f32)), nat.stream())
    nat.check_rc(rc, "omni_tanh_split")
    return out

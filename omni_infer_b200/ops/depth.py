"""Ops of models with norms on both sides of the sublayers, learned positions, and a learned average over depth after every layer.

The residual and the results of the layers are fp32 [T, ld] and [layers + 1, T, ld].  CUDA tensors run
``csrc/kernels/depth_average.cu``, CPU tensors the fp32 references here."""
from __future__ import annotations

import torch

from . import _native as nat
from .layer_list import _f32, _normed_rows, rms_ref


def embed_positions(ids, table, positions, pos_table, x, w, eps, *, ld):
    """x (fp32 [T, ldx], written) = table[ids] + pos_table[positions] (no table: embedding rows alone); returns rmsnorm(x) * w as
    activations [T, ld] with zeros past the width.  Positions past the table add nothing."""
    T, H = ids.shape[0], w.shape[0]
    if not table.is_cuda:
        x[:, :H] = table[ids][:, :H].float()
        if pos_table is not None:
            known = positions < pos_table.shape[0]
            x[:, :H] += pos_table[torch.where(known, positions, 0)][:, :H].float() * known[:, None]
        return _normed_rows(x, w, eps, 1.0, ld, False, table.dtype)
    assert x.dtype == torch.float32 and x.is_contiguous() and x.shape[0] == T
    assert pos_table is None or (pos_table.dtype == table.dtype and pos_table.stride(1) == 1)
    h = torch.empty(T, ld, dtype=table.dtype, device=table.device)
    rc = nat.lib().omni_embed_positions(
        nat.ptr(ids), nat.ptr(table), nat.c_int(table.shape[0]), nat.c_int(table.stride(0)), nat.ptr(positions), nat.ptr(pos_table),
        nat.c_int(pos_table.shape[0] if pos_table is not None else 0), nat.c_int(pos_table.stride(0) if pos_table is not None else 0),
        nat.ptr(x), nat.c_int(T), nat.c_int(H), nat.c_int(x.shape[1]), nat.ptr(w), nat.c_float(eps), nat.ptr(h), nat.c_int(ld),
        nat.c_int(_f32(table)), nat.stream())
    nat.check_rc(rc, "omni_embed_positions")
    return h


def both_norms_step(x_in, x_out, y, w_out, mult, w, eps, dtype, *, ld, results=None, average=None):
    """x_out = x_in + mult * rmsnorm(y) * w_out (fp32; may be in place), returns rmsnorm(x_out) * w as activations [T, ld].

    ``average`` [n + 1] fp32 with ``results`` [>= n + 1, T, ldx]: the sum is also what layer n - 1 gave; it goes to ``results[n]`` (unless
    there is no room for it, after the last layer), and x_out is the sum of ``average[j] * results[j]`` over all n + 1.  ``y``: rows,
    or the parts of an expert mixture (``streams.ExpertSum`` without identity experts)."""
    parts = not torch.is_tensor(y)
    rows = y.y if parts else y
    T, H = x_in.shape[0], w.shape[0]
    n = average.shape[0] - 1 if average is not None else 0
    if not x_in.is_cuda:
        yf = (y.total() if parts else y.float())[:, :H]
        new = x_in[:, :H] + mult * rms_ref(yf, w_out, eps)
        if average is not None:
            if n < results.shape[0]:
                results[n, :, :H] = new
            new = torch.einsum("jtw,j->tw", results[:n, :, :H], average[:n]) + average[n] * new
        x_out[:, :H] = new
        return _normed_rows(x_out, w, eps, 1.0, ld, False, dtype)
    if parts:
        assert y.shared is None or y.shared.stride(0) == rows.stride(0)
    assert rows.dtype == dtype and rows.stride(1) == 1 and x_in.is_contiguous() and x_out.is_contiguous() and x_in.shape == x_out.shape
    assert x_in.dtype == x_out.dtype == w.dtype == w_out.dtype == torch.float32
    assert average is None or (results.is_contiguous() and results.shape[0] >= n and results.shape[1:] == x_in.shape)
    h = torch.empty(T, ld, dtype=dtype, device=x_in.device)
    rc = nat.lib().omni_both_norms_step(
        nat.ptr(x_in), nat.ptr(x_out), nat.c_int(T), nat.c_int(H), nat.c_int(x_in.shape[1]), nat.ptr(rows), nat.c_int(rows.stride(0)),
        nat.ptr(y.row_of if parts else None), nat.c_int(y.ids.shape[1] if parts else 0), nat.ptr(y.shared if parts else None),
        nat.ptr(w_out), nat.c_float(mult), nat.ptr(results if average is not None else None), nat.ptr(average), nat.c_int(n),
        nat.c_int(int(average is not None and n < results.shape[0])), nat.ptr(w), nat.c_float(eps), nat.ptr(h), nat.c_int(ld),
        nat.c_int(int(dtype == torch.float32)), nat.stream())
    nat.check_rc(rc, "omni_both_norms_step")
    return h

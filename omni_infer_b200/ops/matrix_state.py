"""Mixers whose state is a matrix per head, between their projections: the matrix memory of xLSTM (mLSTM), WKV and gated linear
attention (GLA).

CUDA tensors run ``csrc/kernels/matrix_state.cu`` (gates, token by token, norm), ``ssd_sm100.cu`` (mLSTM portions of prompts on
tcgen05) and ``wkv_chunk.cu`` (WKV and GLA portions); CPU tensors the fp32 references here.  Ragged batches as in :mod:`.layer_list`.

State: [slots, H, P, N] fp32 (N key size, P value size; the mLSTM's has one more row, its normaliser) and for the mLSTM
m [slots, H], the running maximum of its log gates.  A request that starts at position 0 starts from zeros."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from . import _native as nat
from .layer_list import _f32, _segments

CHUNK_MIN_ROWS = 8      # portions below this go token by token


@dataclass
class MlstmGates:
    """Per token and head: what the state is kept and a new pair added with, the running maximum, and n . q (filled by the scan).
    ``chunks``: the same per chunk of 128 tokens as the tensor-core form reads it."""
    keep_add: torch.Tensor             # fp32 [T, H, 2]
    m: torch.Tensor                    # fp32 [T, H]
    den: torch.Tensor                  # fp32 [T, H]
    chunks: Optional[torch.Tensor] = None
    n_chunks: int = 0


def mlstm_gates(z, f_col, i_bias, f_bias, cap, m_state, *, positions, state_slots, cu_q=None, chunks=False):
    """z fp32 [T, >= f_col + H]: input gates at column 0, forget gates at ``f_col``, before their biases.  Moves ``m_state``."""
    T, H = z.shape[0], i_bias.shape[0]
    ka = torch.zeros(T, H, 2, dtype=torch.float32, device=z.device)
    m = torch.zeros(T, H, dtype=torch.float32, device=z.device)
    den = torch.zeros(T, H, dtype=torch.float32, device=z.device) if not z.is_cuda else torch.empty_like(m)
    if not z.is_cuda:
        gi = cap * torch.tanh((z[:, :H] + i_bias) / cap)
        gf = F.logsigmoid(cap * torch.tanh((z[:, f_col:f_col + H] + f_bias) / cap))
        for r, a, b in _segments(cu_q, T):
            slot = int(state_slots[r])
            if slot < 0:
                continue
            cur = m_state[slot].clone() if int(positions[a]) > 0 else torch.zeros(H)
            for t in range(a, b):
                new = torch.maximum(gf[t] + cur, gi[t])
                ka[t, :, 0], ka[t, :, 1], m[t] = torch.exp(gf[t] + cur - new), torch.exp(gi[t] - new), new
                cur = new
            m_state[slot] = cur
        return MlstmGates(ka, m, den)
    assert z.dtype == torch.float32 and z.stride(1) == 1
    B = T if cu_q is None else cu_q.shape[0] - 1
    n_chunks = T // 128 + B if chunks and cu_q is not None else 0
    buf = torch.empty(n_chunks * H * (3 * 128 + 5), dtype=torch.float32, device=z.device) if n_chunks else None
    rc = nat.lib().omni_mlstm_gates(
        nat.ptr(z), nat.c_int(z.stride(0)), nat.c_int(f_col), nat.ptr(i_bias), nat.ptr(f_bias), nat.c_float(cap), nat.ptr(m_state),
        nat.ptr(cu_q), nat.ptr(positions), nat.ptr(state_slots), nat.c_int(B), nat.c_int(T), nat.c_int(H), nat.ptr(ka), nat.ptr(m),
        nat.ptr(den), nat.ptr(buf), nat.c_int(n_chunks), nat.stream())
    nat.check_rc(rc, "omni_mlstm_gates")
    return MlstmGates(ka, m, den, buf, n_chunks)


def mlstm_chunked(dtype, N: int, P: int) -> bool:
    """Do portions of prompts run on tensor cores at these sizes?"""
    return dtype == torch.bfloat16 and N % 8 == 0 and N <= 128 and P % 8 == 0


def _tma(*ts) -> bool:
    return all(t.stride(1) == 1 and t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0 for t in ts)


def _rows(kind, a, a_scale, b, v, gates, z, w0, u, state, out, H, P, N, positions, state_slots, cu_q, max_rows, inv_tau=0.0):
    B = a.shape[0] if cu_q is None else cu_q.shape[0] - 1
    rc = nat.lib().omni_state_rows(
        nat.c_int(kind), nat.ptr(a), nat.c_int(a.stride(0)), nat.c_float(a_scale), nat.ptr(b), nat.c_int(b.stride(0)), nat.ptr(v),
        nat.c_int(v.stride(0)), nat.ptr(gates.keep_add if gates else None), nat.ptr(gates.den if gates else None), nat.ptr(z),
        nat.c_int(z.stride(0) if z is not None else 0), nat.ptr(w0), nat.ptr(u), nat.c_float(inv_tau), nat.ptr(state), nat.ptr(cu_q), nat.ptr(positions),
        nat.ptr(state_slots), nat.c_int(B), nat.ptr(out), nat.c_int(out.stride(0)), nat.c_int(H), nat.c_int(P), nat.c_int(N),
        nat.c_int(_f32(a)), nat.c_int(max_rows), nat.stream())
    nat.check_rc(rc, "omni_state_rows")


def mlstm_scan(q, k, v, gates, state, *, H, P, N, positions, state_slots, cu_q=None, min_q=1, max_q=0, by_rows=False):
    """q, k [T, H N], v [T, H P] (rows of any pitch); q is scaled by N^-1/2 here.  Returns S^T q [T, H P], not yet divided by
    the normaliser whose n . q is left in ``gates.den`` (:func:`head_norm` divides)."""
    T, scale = q.shape[0], N ** -0.5
    out = torch.empty(T, H * P, dtype=q.dtype, device=q.device)
    if not q.is_cuda:
        for r, a, b in _segments(cu_q, T):
            slot = int(state_slots[r])
            if slot < 0:
                out[a:b] = 0
                continue
            S = state[slot].clone() if int(positions[a]) > 0 else torch.zeros_like(state[slot])
            for t in range(a, b):
                x = torch.cat([v[t].float().view(H, P), torch.ones(H, 1)], 1)
                S = gates.keep_add[t, :, 0, None, None] * S + (gates.keep_add[t, :, 1, None] * x)[:, :, None] * k[t].float().view(H, 1, N)
                y = torch.einsum("hpn,hn->hp", S, q[t].float().view(H, N) * scale)
                out[t], gates.den[t] = y[:, :P].reshape(-1).to(out.dtype), y[:, P]
            state[slot] = S
        return out
    max_rows = 0
    if cu_q is not None and not by_rows and gates.chunks is not None and mlstm_chunked(q.dtype, N, P) and _tma(q, k, v):
        rc = nat.lib().omni_mlstm_chunks(
            nat.ptr(q), nat.c_int(q.stride(0)), nat.ptr(k), nat.c_int(k.stride(0)), nat.ptr(v), nat.c_int(v.stride(0)), nat.c_int64(T),
            nat.ptr(gates.chunks), nat.c_int(gates.n_chunks), nat.ptr(gates.den), nat.c_float(scale), nat.ptr(state), nat.ptr(cu_q),
            nat.ptr(positions), nat.ptr(state_slots), nat.c_int(cu_q.shape[0] - 1), nat.c_int(max_q or T), nat.ptr(out),
            nat.c_int(out.stride(0)), nat.c_int(H), nat.c_int(P), nat.c_int(N), nat.c_int(CHUNK_MIN_ROWS),
            nat.ptr(nat.status_buffer(q.device)), nat.stream())
        nat.check_rc(rc, "omni_mlstm_chunks")
        if min_q >= CHUNK_MIN_ROWS:
            return out
        max_rows = CHUNK_MIN_ROWS - 1
    _rows(0, q, scale, k, v, gates, None, None, None, state, out, H, P, N, positions, state_slots, cu_q, max_rows)
    return out


def wkv_scan(r, k, v, z, w0, u, state, *, H, N, positions, state_slots, cu_q=None, min_q=1, max_q=0, by_rows=False):
    """r, k, v [T, H N], z fp32 [T, H N] (rows of any pitch), the decay being exp(-exp(z + w0)) -> o [T, H N]."""
    T = r.shape[0]
    out = torch.empty(T, H * N, dtype=r.dtype, device=r.device)
    if not r.is_cuda:
        w = torch.exp(-torch.exp(z[:, :H * N].float() + w0)).view(T, H, 1, N)
        for q, a, b in _segments(cu_q, T):
            slot = int(state_slots[q])
            if slot < 0:
                out[a:b] = 0
                continue
            S = state[slot].clone() if int(positions[a]) > 0 else torch.zeros_like(state[slot])      # [H, P, N]
            for t in range(a, b):
                kv = v[t].float().view(H, N, 1) * k[t].float().view(H, 1, N)
                out[t] = torch.einsum("hpn,hn->hp", S + u.view(H, 1, N) * kv, r[t].float().view(H, N)).reshape(-1).to(out.dtype)
                S = w[t] * S + kv
            state[slot] = S
        return out
    assert z.dtype == torch.float32
    max_rows = 0
    if cu_q is not None and not by_rows and r.dtype == torch.bfloat16 and N % 8 == 0 and N <= 128 and _tma(v):
        rc = nat.lib().omni_wkv_chunks(
            nat.ptr(r), nat.c_int(r.stride(0)), nat.ptr(k), nat.c_int(k.stride(0)), nat.ptr(v), nat.c_int(v.stride(0)), nat.ptr(z),
            nat.c_int(z.stride(0)), nat.ptr(w0), nat.ptr(u), nat.ptr(state), nat.ptr(cu_q), nat.ptr(positions), nat.ptr(state_slots),
            nat.c_int(cu_q.shape[0] - 1), nat.c_int(max_q or T), nat.ptr(out), nat.c_int(out.stride(0)), nat.c_int(H), nat.c_int(N),
            nat.c_int(CHUNK_MIN_ROWS), nat.ptr(nat.status_buffer(r.device)), nat.stream())
        nat.check_rc(rc, "omni_wkv_chunks")
        if min_q >= CHUNK_MIN_ROWS:
            return out
        max_rows = CHUNK_MIN_ROWS - 1
    _rows(1, r, 1.0, k, v, None, z, w0, u, state, out, H, N, N, positions, state_slots, cu_q, max_rows)
    return out


def gla_chunked(dtype, N: int, P: int) -> bool:
    """Do portions of prompts run in chunks at these sizes?"""
    return dtype == torch.bfloat16 and N % 8 == 0 and N <= 256 and P % 8 == 0


def gla_scan(q, k, v, z, bias, inv_tau, state, *, H, P, N, positions, state_slots, cu_q=None, min_q=1, max_q=0, by_rows=False):
    """S <- diag(a) S + k v^T, o = S^T q N^-1/2 with a = sigmoid(z + bias)^inv_tau per head and key channel; q, k [T, H N],
    v [T, H P], z fp32 [T, >= H N] (rows of any pitch) -> o [T, H P]."""
    T, scale = q.shape[0], N ** -0.5
    out = torch.empty(T, H * P, dtype=q.dtype, device=q.device)
    if not q.is_cuda:
        a = torch.exp(F.logsigmoid(z[:, :H * N].float() + bias) * inv_tau).view(T, H, 1, N)
        for r, first, end in _segments(cu_q, T):
            slot = int(state_slots[r])
            if slot < 0:
                out[first:end] = 0
                continue
            S = state[slot].clone() if int(positions[first]) > 0 else torch.zeros_like(state[slot])      # [H, P, N]
            for t in range(first, end):
                S = a[t] * S + v[t].float().view(H, P, 1) * k[t].float().view(H, 1, N)
                out[t] = torch.einsum("hpn,hn->hp", S, q[t].float().view(H, N) * scale).reshape(-1).to(out.dtype)
            state[slot] = S
        return out
    assert z.dtype == torch.float32 and z.stride(1) == 1 and state.dtype == torch.float32
    max_rows = 0
    if cu_q is not None and not by_rows and gla_chunked(q.dtype, N, P) and _tma(v):
        rc = nat.lib().omni_gla_chunks(
            nat.ptr(q), nat.c_int(q.stride(0)), nat.ptr(k), nat.c_int(k.stride(0)), nat.ptr(v), nat.c_int(v.stride(0)), nat.ptr(z),
            nat.c_int(z.stride(0)), nat.ptr(bias), nat.c_float(scale), nat.c_float(inv_tau), nat.ptr(state), nat.ptr(cu_q),
            nat.ptr(positions), nat.ptr(state_slots), nat.c_int(cu_q.shape[0] - 1), nat.c_int(max_q or T), nat.ptr(out),
            nat.c_int(out.stride(0)), nat.c_int(H), nat.c_int(P), nat.c_int(N), nat.c_int(CHUNK_MIN_ROWS),
            nat.ptr(nat.status_buffer(q.device)), nat.stream())
        nat.check_rc(rc, "omni_gla_chunks")
        if min_q >= CHUNK_MIN_ROWS:
            return out
        max_rows = CHUNK_MIN_ROWS - 1
    _rows(2, q, scale, k, v, None, z, bias, None, state, out, H, P, N, positions, state_slots, cu_q, max_rows, inv_tau)
    return out


def head_norm(y, gate, w, out, *, H, P, eps, act, scale=1.0, gates=None):
    """out[:, :H P] = y of every head over its root mean square, times ``w``, ``act(gate)`` ("sigmoid" | "silu") and ``scale``.
    ``gates``: y is divided by max(|n . q|, exp(-m)) + 1e-6 first."""
    T = y.shape[0]
    if not y.is_cuda:
        o = y.float().view(T, H, P)
        if gates is not None:
            o = o / (torch.maximum(gates.den.abs(), torch.exp(-gates.m)) + 1e-6).unsqueeze(-1)
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
        g = gate[:, :H * P].float()
        g = torch.sigmoid(g) if act == "sigmoid" else F.silu(g)
        out[:, :H * P] = (o.reshape(T, H * P) * w * g * scale).to(out.dtype)
        return out
    rc = nat.lib().omni_head_norm(
        nat.ptr(y), nat.c_int(y.stride(0)), nat.ptr(gates.den if gates else None), nat.ptr(gates.m if gates else None), nat.ptr(gate),
        nat.c_int(gate.stride(0)), nat.ptr(w), nat.c_float(scale), nat.ptr(out), nat.c_int(out.stride(0)), nat.c_int(T), nat.c_int(H),
        nat.c_int(P), nat.c_float(eps), nat.c_int(0 if act == "sigmoid" else 1), nat.c_int(_f32(y)), nat.stream())
    nat.check_rc(rc, "omni_head_norm")
    return out

"""Ops of the layer-list models: the fp32 residual stream with norms on the sublayers' outputs or ahead of the sublayers, attention
over the paged cache (windows, kept first tokens, chunks, capped and biased scores) with a q/k norm over the whole projection, the
short convolution, and the Mamba-2 layer between its projections.

CUDA tensors run ``csrc/kernels/post_norm_ops.cu``, ``attn_any.cu``, ``fmha_sm100.cu``, ``gqa_decode.cu``, ``short_conv.cu`` and
``mamba2.cu`` / ``ssd_sm100.cu``; CPU tensors run the fp32 references here.  Activations are bf16 or fp32.  Rows may be wider than their
content (a multiple of 8 columns, so that they can be TMA operands); the columns past it are zero.

Ragged batches: the rows of request r are ``cu_q[r]:cu_q[r + 1]``, its rows' positions ascend by one, ``q_to_seq[row] = r``.
``cu_q=None``: one row per request (decode)."""
from __future__ import annotations

import torch
import torch.nn.functional as F

from . import _native as nat
from .gemm import clamped_glu_ref


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _f32(t) -> int:
    assert t.dtype in (torch.float32, torch.bfloat16)
    return int(t.dtype == torch.float32)


def _segments(cu_q, rows: int):
    """(request, first row, end row) of every request with rows."""
    if cu_q is None:
        return [(i, i, i + 1) for i in range(rows)]
    c = cu_q.tolist()
    return [(i, c[i], c[i + 1]) for i in range(len(c) - 1) if c[i + 1] > c[i]]


# ----------------------------------------------------------------------------- residual stream
def embed_residual(ids, table):
    """Embedding rows -> (fp32 residual, activations).  fp32 activations are the residual itself."""
    if not table.is_cuda:
        x = table[ids].float()
        return x, (x if table.dtype == torch.float32 else x.to(table.dtype))
    T, ld = ids.shape[0], table.shape[1]
    x = torch.empty(T, ld, dtype=torch.float32, device=table.device)
    xa = None if table.dtype == torch.float32 else torch.empty(T, ld, dtype=table.dtype, device=table.device)
    rc = nat.lib().omni_embed_residual(nat.ptr(ids), nat.ptr(table), nat.c_int(table.shape[0]), nat.c_int(T), nat.c_int(ld),
                                       nat.ptr(x), nat.ptr(xa), nat.c_int(_f32(table)), nat.stream())
    nat.check_rc(rc, "omni_embed_residual")
    return x, (x if xa is None else xa)


def rms_ref(x, w, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def post_norm_add(y, w, x, eps):
    """x (fp32, in place) += rmsnorm(y) * w; returns the activations for the next sublayer (x itself in fp32 runs)."""
    H = w.shape[0]
    f32 = y.dtype == torch.float32
    if not y.is_cuda:
        x[:, :H] += rms_ref(y[:, :H].float(), w, eps)
        return x if f32 else x.to(y.dtype)
    assert x.dtype == torch.float32 and w.dtype == torch.float32 and y.stride(1) == 1 and x.is_contiguous()
    xa = None if f32 else torch.empty(x.shape, dtype=y.dtype, device=y.device)
    rc = nat.lib().omni_post_norm_add(nat.ptr(y), nat.c_int(y.stride(0)), nat.ptr(w), nat.ptr(x), nat.ptr(xa),
                                      nat.c_int(y.shape[0]), nat.c_int(H), nat.c_int(x.shape[1]), nat.c_float(eps),
                                      nat.c_int(_f32(y)), nat.stream())
    nat.check_rc(rc, "omni_post_norm_add")
    return x if f32 else xa


def rmsnorm_residual(x, w, eps, dtype):
    """Norm of the fp32 residual, as activations of ``dtype``."""
    H = w.shape[0]
    if not x.is_cuda:
        out = torch.zeros(x.shape, dtype=dtype)
        out[:, :H] = rms_ref(x[:, :H], w, eps).to(dtype)
        return out
    out = torch.empty(x.shape, dtype=dtype, device=x.device)
    rc = nat.lib().omni_rmsnorm_residual(nat.ptr(x), nat.ptr(w), nat.ptr(out), nat.c_int(x.shape[0]), nat.c_int(H),
                                         nat.c_int(x.shape[1]), nat.c_float(eps), nat.c_int(_f32(out)), nat.stream())
    nat.check_rc(rc, "omni_rmsnorm_residual")
    return out


def _normed_rows(x, w, eps, scale, ld, ones, dtype):
    H = w.shape[0]
    h = torch.zeros(x.shape[0], ld, dtype=dtype)
    h[:, :H] = (rms_ref(x[:, :H], w, eps) * scale).to(dtype)
    if ones:
        h[:, H] = 1
    return h


def _residual_call(x, w, eps, scale, ld, ones, dtype, ids=None, table=None, y=None, bias=None):
    """``y``: rows, or the parts of an expert mixture (``streams.ExpertSum`` without identity experts)."""
    parts = y is not None and not torch.is_tensor(y)
    rows = y.y if parts else y
    if parts:
        assert y.shared is None or y.shared.stride(0) == rows.stride(0)
    assert x.dtype == torch.float32 and w.dtype == torch.float32 and x.is_contiguous() and (rows is None or (rows.dtype == dtype and rows.stride(1) == 1))
    T, H = x.shape[0], w.shape[0]
    h = torch.empty(T, ld, dtype=dtype, device=x.device)
    rc = nat.lib().omni_residual_norm(
        nat.ptr(x), nat.c_int(T), nat.c_int(H), nat.c_int(x.shape[1]), nat.ptr(ids), nat.ptr(table),
        nat.c_int(table.shape[0] if table is not None else 0), nat.c_int(table.stride(0) if table is not None else 0), nat.ptr(rows),
        nat.c_int(rows.stride(0) if rows is not None else 0), nat.ptr(y.row_of if parts else None),
        nat.c_int(y.ids.shape[1] if parts else 0), nat.ptr(y.shared if parts else None), nat.ptr(bias), nat.ptr(w), nat.c_float(eps),
        nat.c_float(scale), nat.ptr(h), nat.c_int(ld), nat.c_int(int(ones)), nat.c_int(int(dtype == torch.float32)), nat.stream())
    nat.check_rc(rc, "omni_residual_norm")
    return h


def embed_norm(ids, table, w, eps, *, ld, ones=False):
    """Embedding rows -> (fp32 residual, rmsnorm of it times ``w`` as activations [T, ld]).  Columns past the width are zeros, but
    for the first of them with ``ones`` (it meets the column of the next weight that holds the biases)."""
    T, H = ids.shape[0], w.shape[0]
    x = torch.empty(T, pad8(H), dtype=torch.float32, device=table.device)
    if not table.is_cuda:
        x[:, :H] = table[ids][:, :H].float()
        return x, _normed_rows(x, w, eps, 1.0, ld, ones, table.dtype)
    return x, _residual_call(x, w, eps, 1.0, ld, ones, table.dtype, ids=ids, table=table)


def add_norm(x, y, w, eps, dtype, *, ld, ones=False, bias=None, scale=1.0):
    """x (fp32, in place) += y + bias, then as :func:`embed_norm`; ``scale`` multiplies the normed rows."""
    if not x.is_cuda:
        H = w.shape[0]
        x[:, :H] += (y.float() if torch.is_tensor(y) else y.total())[:, :H]
        if bias is not None:
            x[:, :H] += bias
        return _normed_rows(x, w, eps, scale, ld, ones, dtype)
    return _residual_call(x, w, eps, scale, ld, ones, dtype, y=y, bias=bias)


# ----------------------------------------------------------------------------- q/k norm, rotation, cache write
def _rotate_half_ref(x, cos_sin, positions, rot):
    """x [T, heads, D] fp32; rotates the first ``rot`` entries of every head."""
    if rot == 0:
        return x
    cs = cos_sin[positions]
    c, s = cs[:, None, : rot // 2], cs[:, None, rot // 2:]
    u, v = x[..., : rot // 2], x[..., rot // 2: rot]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., rot:]], -1)


def qk_norm_rope_cache(qkv, hq, hkv, dk, dv, q_w, k_w, eps, cos_sin, rot, positions, slots, k_cache, v_cache):
    """``qkv`` rows are q heads | k heads | v heads (``hkv=0``: q only).  RMSNorm over the whole q and the whole k
    projection (``q_w=None``: none), rotate-half RoPE on the first ``rot`` dimensions of every head; q in place, k and v into the caches
    [blocks, block, hkv, d] at ``slots`` (-1: not stored)."""
    T, nq, nk = qkv.shape[0], hq * dk, hkv * dk
    if not qkv.is_cuda:
        norm = (lambda x, w: x) if q_w is None else (lambda x, w: rms_ref(x, w, eps))
        q = norm(qkv[:, :nq].float(), q_w).view(T, hq, dk)
        qkv[:, :nq] = _rotate_half_ref(q, cos_sin, positions, rot).reshape(T, nq).to(qkv.dtype, copy=True)
        if hkv:
            k = norm(qkv[:, nq:nq + nk].float(), k_w).view(T, hkv, dk)
            k = _rotate_half_ref(k, cos_sin, positions, rot)
            ok = slots >= 0
            k_cache.view(-1, hkv, dk)[slots[ok]] = k[ok].to(k_cache.dtype)
            v_cache.view(-1, hkv, dv)[slots[ok]] = qkv[:, nq + nk:nq + nk + hkv * dv].view(T, hkv, dv)[ok]
        return
    assert qkv.stride(1) == 1 and (not hkv or k_cache.dtype == qkv.dtype)
    rc = nat.lib().omni_qk_norm_rope_cache(
        nat.ptr(qkv), nat.c_int(qkv.stride(0)), nat.c_int(hq), nat.c_int(hkv), nat.c_int(dk), nat.c_int(dv), nat.ptr(q_w),
        nat.ptr(k_w), nat.c_float(eps), nat.ptr(cos_sin), nat.c_int(rot), nat.ptr(positions), nat.ptr(slots),
        nat.ptr(k_cache if hkv else None), nat.ptr(v_cache if hkv else None), nat.c_int(T), nat.c_int(_f32(qkv)), nat.stream())
    nat.check_rc(rc, "omni_qk_norm_rope_cache")


# ----------------------------------------------------------------------------- windowed attention over the paged cache
def first_visible(pos: int, window: int, chunk: int) -> int:
    """First key that a query at ``pos`` sees through its window and in its chunk (0: none)."""
    return max(0, pos - window + 1 if window else 0, pos // chunk * chunk if chunk else 0)


def paged_attention_ref(q, k_cache, v_cache, positions, q_to_seq, slots, block_table, scale, window, sink, out_scale, out, keep_first=0,
                        chunk=0, softcap=0.0, slopes=None, gate=None, log_bias=None):
    hq, dk = q.shape[1], q.shape[2]
    bs, hkv, dv = k_cache.shape[1], k_cache.shape[2], v_cache.shape[3]
    kf, vf = k_cache.flatten(0, 1), v_cache.flatten(0, 1)
    rep = hq // hkv
    out[:, :hq * dv] = 0
    for t in range(q.shape[0]):
        if int(slots[t]) < 0:
            continue
        p = int(positions[t])
        lo = first_visible(p, window, chunk)
        pos = torch.cat([torch.arange(min(keep_first, lo)), torch.arange(lo, p + 1)])
        rows = block_table[int(q_to_seq[t]), pos // bs].long() * bs + pos % bs
        k = kf[rows].float().repeat_interleave(rep, 1)
        v = vf[rows].float().repeat_interleave(rep, 1)
        s = torch.einsum("hd,lhd->hl", q[t].float(), k) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if slopes is not None:
            s = s - slopes[:, None] * (p - pos)
        if log_bias is not None:
            s = s - log_bias[0][:, None] * torch.log1p(log_bias[1][:, None] * (p - pos))
        if sink is not None:
            s = torch.cat([s, sink[:, None]], 1)
        o = torch.einsum("hl,lhd->hd", torch.softmax(s, -1)[:, :len(pos)], v) * out_scale
        if gate is not None:
            o = o * torch.sigmoid(gate[t].float()).view(hq, -1)
        out[t, :hq * dv] = o.reshape(-1).to(out.dtype)
    return out


def _splits(ctas: int, keys: int) -> int:
    """Parts of the key range of a decode launch with that many blocks: three of them fit an SM, and a part should have several
    tiles of 32 keys per warp."""
    tiles = (keys + 31) // 32 + 1
    return max(1, min((444 + ctas - 1) // ctas, tiles // 8, 32)) if ctas < 444 else 1


def paged_attention(q, k_cache, v_cache, *, positions, q_to_seq, slots, block_table, seq_lens, scale, window=0, cu_q=None,
                    max_q=1, max_seq_len=0, sink=None, out_scale=1.0, out=None, any_shape=False, keep_first=0, chunk=0, softcap=0.0,
                    slopes=None, gate=None, rows_share=False, log_bias=None):
    """q [T, hq, dk] (rows of any pitch) against the cached keys of the rows' requests, each row seeing the ``window``
    positions up to its own (0: all of them), only those of its own ``chunk`` of positions (0: no chunks), and the ``keep_first``
    first ones in any case.  A score is ``softcap tanh(q k scale / softcap) - slopes[head] distance``, less ``r1[head]
    ln(1 + r2[head] distance)`` with ``log_bias`` = (r1, r2) (each part optional).  ``sink`` [hq] fp32: exp(sink) is one more term of
    the head's softmax denominator; ``out_scale`` multiplies the result, and so does the sigmoid of ``gate``, [T, hq]
    or [T, hq * dv].  Returns [T, pad8(hq * dv)], or writes the first columns of ``out``.  The value cache may be a
    column slice of the key cache (one key/value head).

    bf16 portions of prompts run on tcgen05 (``omni_fmha_paged``), bf16 single tokens on the split-KV decode kernel; fp32
    and head shapes those two do not take - or ``any_shape`` - go to ``omni_attn_any``.  ``cu_q=None``: every row stands alone;
    with ``rows_share`` they belong to the requests ``q_to_seq`` (else row i to request i) and see ``seq_lens`` keys each."""
    T, hq, dk = q.shape
    bs, hkv, dv = k_cache.shape[1], k_cache.shape[2], v_cache.shape[3]
    if out is None:
        ld = pad8(hq * dv)
        out = (torch.empty if ld == hq * dv else torch.zeros)(T, ld, dtype=q.dtype, device=q.device)
    ld = out.stride(0)
    if not q.is_cuda:
        return paged_attention_ref(q, k_cache, v_cache, positions, q_to_seq, slots, block_table, scale, window, sink, out_scale, out,
                                   keep_first, chunk, softcap, slopes, gate, log_bias)
    assert q.stride(2) == 1 and q.stride(1) == dk and k_cache.dtype == q.dtype and block_table.stride(1) == 1
    k_row, v_row = k_cache.stride(1), v_cache.stride(1)
    assert k_cache.stride(0) == bs * k_row and v_cache.stride(0) == bs * v_row
    assert gate is None or (gate.dtype == q.dtype and gate.stride(1) == 1 and gate.shape[1] in (hq, hq * dv))
    r1, r2 = log_bias if log_bias is not None else (None, None)
    packed = k_row == hkv * dk and v_row == hkv * dv
    f32 = _f32(q)
    lib = nat.lib()
    gate_args = (nat.ptr(gate), nat.c_int(gate.stride(0) if gate is not None else 0), nat.c_int(gate.shape[1] // hq if gate is not None else 1))
    mod = (nat.c_int(window), nat.c_int(chunk), nat.c_int(keep_first), nat.c_float(scale), nat.c_float(softcap), nat.ptr(slopes), nat.ptr(r1),
           nat.ptr(r2), nat.ptr(sink))
    tc = not any_shape and not f32 and ld % 8 == 0 and out.data_ptr() % 16 == 0 and dk % 8 == 0 and dv % 8 == 0 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0
    vec_gate = gate is None or (gate.shape[1] == hq * dv and gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0)
    if tc and cu_q is not None and dk <= 192 and dv <= 128 and bs % 64 == 0 and packed and vec_gate and scale > 0:
        rc = lib.omni_fmha_paged(
            nat.ptr(q), nat.c_int64(T), nat.c_int(q.stride(0)), nat.ptr(k_cache), nat.ptr(v_cache),
            nat.c_int64(k_cache.shape[0] * bs), nat.ptr(cu_q), nat.ptr(seq_lens), nat.ptr(block_table),
            nat.c_int(block_table.stride(0)), nat.c_int(cu_q.shape[0] - 1), nat.c_int(max_q), nat.c_int(hq), nat.c_int(hkv),
            nat.c_int(dk), nat.c_int(dv), nat.c_int(bs), *mod, *gate_args[:2], nat.c_float(out_scale), nat.ptr(out), nat.c_int(ld),
            nat.ptr(nat.status_buffer(q.device)), nat.stream())
        nat.check_rc(rc, "omni_fmha_paged")
        return out
    if tc and cu_q is None and dk <= 256 and dv <= 256 and k_row % 8 == 0 and v_row % 8 == 0:
        span = min(max_seq_len, window + keep_first if window else max_seq_len, chunk + keep_first if chunk else max_seq_len)
        splits = _splits(T * hkv * ((hq // hkv + 15) // 16), span)
        o_part = lse = None
        if splits > 1:
            o_part = torch.empty(T * splits * hq * dv, dtype=torch.float32, device=q.device)
            lse = torch.empty(T * splits * hq, dtype=torch.float32, device=q.device)
        rc = lib.omni_gqa_paged_decode_window(
            nat.ptr(q), nat.c_int(q.stride(0)), nat.ptr(k_cache), nat.ptr(v_cache), nat.c_int64(k_row), nat.c_int64(v_row),
            nat.ptr(q_to_seq if rows_share else None), nat.ptr(block_table), nat.c_int(block_table.stride(0)), nat.ptr(seq_lens),
            nat.c_int(T), nat.c_int(hq), nat.c_int(hkv), nat.c_int(dk), nat.c_int(dv), nat.c_int(bs), *mod, *gate_args,
            nat.c_float(out_scale), nat.c_int(splits), nat.ptr(o_part), nat.ptr(lse), nat.ptr(out), nat.c_int(ld), nat.stream())
        nat.check_rc(rc, "omni_gqa_paged_decode_window")
        return out
    rc = lib.omni_attn_any(
        nat.ptr(q), nat.c_int(q.stride(0)), nat.ptr(k_cache), nat.ptr(v_cache), nat.c_int64(k_row), nat.c_int64(v_row),
        nat.ptr(positions), nat.ptr(q_to_seq), nat.ptr(slots), nat.ptr(block_table), nat.c_int(block_table.stride(0)), nat.c_int(T),
        nat.c_int(hq), nat.c_int(hkv), nat.c_int(dk), nat.c_int(dv), nat.c_int(bs), *mod, *gate_args, nat.c_float(out_scale),
        nat.ptr(out), nat.c_int(ld), nat.c_int(f32), nat.stream())
    nat.check_rc(rc, "omni_attn_any")
    return out


# ----------------------------------------------------------------------------- gated feed-forward
def gated_mul(x, inter, up_off, kind="geglu", limit=0.0):
    """act(x[:, :inter], x[:, up_off:up_off + inter]) -> [T, pad8(inter)]; kinds as the gated epilogues of ``ops.gemm``."""
    T, ld = x.shape[0], pad8(inter)
    if not x.is_cuda:
        g, u = x[:, :inter].float(), x[:, up_off:up_off + inter].float()
        y = clamped_glu_ref(g, u, limit) if kind == "clamped_glu" else (F.silu(g) if kind == "swiglu" else F.gelu(g, approximate="tanh")) * u
        return F.pad(y, (0, ld - inter)).to(x.dtype)
    out = torch.empty(T, ld, dtype=x.dtype, device=x.device)
    rc = nat.lib().omni_gated_mul(nat.ptr(x), nat.c_int(x.stride(0)), nat.c_int(up_off), nat.ptr(out), nat.c_int(ld),
                                  nat.c_int(T), nat.c_int(inter), nat.c_int({"geglu": 0, "clamped_glu": 1, "swiglu": 2}[kind]),
                                  nat.c_float(limit), nat.c_int(_f32(x)), nat.stream())
    nat.check_rc(rc, "omni_gated_mul")
    return out


# ----------------------------------------------------------------------------- short convolution
def short_conv_ref(u, w, bias, state, positions, state_slots, cu_q, out, silu):
    taps, C = w.shape
    for r, a, b in _segments(cu_q, u.shape[0]):
        slot = int(state_slots[r])
        if slot < 0:
            out[a:b, :C] = 0
            continue
        old = state[slot].float() if taps > 1 else u.new_zeros(0, C).float()
        pos0 = int(positions[a])
        if pos0 < taps - 1:                       # entries before the start of the sequence
            old = old.clone()
            old[: taps - 1 - pos0] = 0
        full = torch.cat([old, u[a:b, :C].float()])
        y = sum(full[k:k + b - a] * w[k] for k in range(taps))
        if bias is not None:
            y = y + bias
        out[a:b, :C] = (F.silu(y) if silu else y).to(out.dtype)
        if taps > 1:
            state[slot] = full[b - a:].to(state.dtype)
    return out


def short_conv(u, w, bias, state, *, positions, state_slots, q_to_seq=None, cu_q=None, silu=False):
    """Causal convolution per channel (``w`` [taps, C], last tap = current token), bias (or None), optionally silu.  u [T, C] (rows
    of any pitch); ``state`` [slots, taps - 1, C] holds the last inputs of every request and is moved on.  -> [T, pad8(C)]."""
    T, (taps, C) = u.shape[0], w.shape
    out = torch.empty(T, pad8(C), dtype=u.dtype, device=u.device)
    if not u.is_cuda:
        return short_conv_ref(u, w, bias, state, positions, state_slots, cu_q, out, silu)
    assert u.stride(1) == 1 and state.dtype == u.dtype and w.is_contiguous()
    B = T if cu_q is None else cu_q.shape[0] - 1
    rc = nat.lib().omni_short_conv(
        nat.ptr(u), nat.c_int(u.stride(0)), nat.c_int(C), nat.c_int(taps), nat.ptr(w), nat.ptr(bias), nat.ptr(state),
        nat.ptr(positions), nat.ptr(q_to_seq), nat.ptr(cu_q), nat.ptr(state_slots), nat.c_int(B), nat.c_int(T), nat.ptr(out),
        nat.c_int(out.shape[1]), nat.c_int(int(silu)), nat.c_int(_f32(u)), nat.stream())
    nat.check_rc(rc, "omni_short_conv")
    return out


def conv_silu(u, w, bias, state, **where):
    """:func:`short_conv` with a silu on its output, as Mamba-2 has it."""
    return short_conv(u, w, bias, state, silu=True, **where)


# ----------------------------------------------------------------------------- Mamba-2
def ssm_scan_ref(xbc, dt, A_log, dt_bias, D, state, positions, state_slots, cu_q, H, P, N, G, out):
    inner = H * P
    of = torch.arange(H) // (H // G)
    A = -torch.exp(A_log)
    for r, a, b in _segments(cu_q, xbc.shape[0]):
        slot = int(state_slots[r])
        if slot < 0:
            out[a:b] = 0
            continue
        S = state[slot] if int(positions[a]) > 0 else torch.zeros_like(state[slot])      # [H, P, N]
        for t in range(a, b):
            x = xbc[t, :inner].float().view(H, P)
            B = xbc[t, inner:inner + G * N].float().view(G, N)[of]
            C = xbc[t, inner + G * N:inner + 2 * G * N].float().view(G, N)[of]
            d = F.softplus(dt[t].float() + dt_bias, threshold=1e9)
            S = torch.exp(A * d)[:, None, None] * S + (d[:, None] * x)[:, :, None] * B[:, None, :]
            y = torch.einsum("hpn,hn->hp", S, C) + D[:, None] * x
            out[t, :inner] = y.reshape(-1).to(out.dtype)
        state[slot] = S
    return out


SSD_MIN_ROWS = 8      # portions below this go token by token: a chunk of the tensor-core form costs as much as some tokens


def ssm_scan(xbc, dt, A_log, dt_bias, D, state, *, H, P, N, G, positions, state_slots, cu_q=None, min_q=1, max_q=0, by_rows=False):
    """S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x with dt = softplus(dt + dt_bias), per head; ``xbc`` rows are
    x | B | C, ``dt`` [T, H] (rows of any pitch), ``state`` [slots, H, P, N] fp32.  Requests that start at position 0 start
    from zeros.  ``min_q`` / ``max_q``: rows of the shortest / longest request, if known.  ``by_rows``: token by token even where the chunked
    tensor-core forms apply.  -> y [T, pad8(H P)]."""
    T = xbc.shape[0]
    out = torch.empty(T, pad8(H * P), dtype=xbc.dtype, device=xbc.device)
    if not xbc.is_cuda:
        return ssm_scan_ref(xbc, dt, A_log, dt_bias, D, state, positions, state_slots, cu_q, H, P, N, G, out)
    assert xbc.stride(1) == 1 and dt.dtype == xbc.dtype and dt.stride(1) == 1 and state.dtype == torch.float32
    B = T if cu_q is None else cu_q.shape[0] - 1
    max_rows = -1 if by_rows else 0
    if (cu_q is not None and not by_rows and xbc.dtype == torch.bfloat16 and P % 8 == 0 and N % 8 == 0 and N <= 128
            and xbc.stride(0) % 8 == 0 and xbc.data_ptr() % 16 == 0):
        scratch = torch.empty(3 * (T // 128 + B) * H * 128, dtype=torch.float32, device=xbc.device)
        rc = nat.lib().omni_ssd_chunks(
            nat.ptr(xbc), nat.c_int(xbc.stride(0)), nat.c_int64(T), nat.ptr(dt), nat.c_int(dt.stride(0)), nat.ptr(A_log),
            nat.ptr(dt_bias), nat.ptr(D), nat.ptr(state), nat.ptr(cu_q), nat.ptr(positions), nat.ptr(state_slots),
            nat.c_int(B), nat.c_int(max_q or T), nat.ptr(out), nat.c_int(out.stride(0)), nat.c_int(H), nat.c_int(P), nat.c_int(N),
            nat.c_int(G), nat.c_int(SSD_MIN_ROWS), nat.ptr(scratch), nat.ptr(nat.status_buffer(xbc.device)), nat.stream())
        nat.check_rc(rc, "omni_ssd_chunks")
        if min_q >= SSD_MIN_ROWS:
            return out
        max_rows = SSD_MIN_ROWS - 1
    rc = nat.lib().omni_ssm_scan(
        nat.ptr(xbc), nat.c_int(xbc.stride(0)), nat.ptr(dt), nat.c_int(dt.stride(0)), nat.ptr(A_log), nat.ptr(dt_bias),
        nat.ptr(D), nat.ptr(state), nat.ptr(cu_q), nat.ptr(positions), nat.ptr(state_slots), nat.c_int(B), nat.ptr(out),
        nat.c_int(out.stride(0)), nat.c_int(H), nat.c_int(P), nat.c_int(N), nat.c_int(G), nat.c_int(_f32(xbc)),
        nat.c_int(max_rows), nat.stream())
    nat.check_rc(rc, "omni_ssm_scan")
    return out


def gated_group_norm(y, z, w, parts, eps):
    """RMSNorm of y * silu(z) in ``parts`` equal parts, times w.  y, z: rows of at least len(w) columns."""
    T, inner = y.shape[0], w.shape[0]
    ld = pad8(inner)
    if not y.is_cuda:
        g = y[:, :inner].float() * F.silu(z[:, :inner].float())
        g = g.view(T, parts, -1)
        g = g * torch.rsqrt(g.pow(2).mean(-1, keepdim=True) + eps)
        return F.pad(g.reshape(T, inner) * w, (0, ld - inner)).to(y.dtype)
    out = torch.empty(T, ld, dtype=y.dtype, device=y.device)
    rc = nat.lib().omni_gated_group_norm(
        nat.ptr(y), nat.c_int(y.stride(0)), nat.ptr(z), nat.c_int(z.stride(0)), nat.ptr(w), nat.ptr(out), nat.c_int(ld),
        nat.c_int(T), nat.c_int(inner), nat.c_int(parts), nat.c_float(eps), nat.c_int(_f32(y)), nat.stream())
    nat.check_rc(rc, "omni_gated_group_norm")
    return out

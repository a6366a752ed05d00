"""Ops between the input projections of an attention layer and the attention itself - head norms, rotation, value mixing, the
cache write - and the attention over cached latents.

CUDA tensors run ``csrc/kernels/attn_prepare.cu``, ``mla_decode.cu``, ``gqa_decode.cu``, ``fmha_sm100.cu`` and ``attn_any.cu``; CPU
tensors the fp32 references here."""
from __future__ import annotations

import torch

from . import _native as nat
from .layer_list import _f32, _rotate_half_ref, paged_attention, rms_ref


def _rotate_pairs_ref(x, cos_sin, positions, rot):
    """x [T, heads, D] fp32; rotates neighbouring dimensions of the first ``rot`` entries of every head."""
    if rot == 0:
        return x
    cs = cos_sin[positions]
    c, s = cs[:, None, : rot // 2], cs[:, None, rot // 2:]
    u, v = x[..., 0:rot:2], x[..., 1:rot:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., rot:]], -1)


def qkv_prepare(qkv, hq, hkv, dk, dv, q_w, k_w, eps, cos_sin, rot, pairs, positions, slots, k_cache, v_cache, mix=None, v_first=None,
                v_norm=False):
    """``qkv`` rows are q heads | k heads | v heads.  RMSNorm of every q and k head with one weight for all (``q_w=None``: none),
    rotation of the first ``rot`` dimensions of every head (``pairs``: neighbours, else halves); q in place, k and v into the caches
    [blocks, block, hkv, d] at ``slots`` (-1: not stored).  ``mix`` (one value) with ``v_first`` [T, hkv dv]: (1 - mix) v + mix v_first
    is stored; ``v_norm``: every v head divided by its root mean square (not both)."""
    assert not (v_norm and mix is not None)
    T, nq, nk, nv = qkv.shape[0], hq * dk, hkv * dk, hkv * dv
    if not qkv.is_cuda:
        turn = _rotate_pairs_ref if pairs else _rotate_half_ref
        norm = (lambda x, w: x) if q_w is None else (lambda x, w: rms_ref(x, w, eps))
        q = turn(norm(qkv[:, :nq].float().view(T, hq, dk), q_w), cos_sin, positions, rot)
        qkv[:, :nq] = q.reshape(T, nq).to(qkv.dtype, copy=True)
        k = turn(norm(qkv[:, nq:nq + nk].float().view(T, hkv, dk), k_w), cos_sin, positions, rot)
        v = qkv[:, nq + nk:nq + nk + nv].float()
        if mix is not None:
            v = (1 - mix) * v + mix * v_first.float()
        if v_norm:
            v = rms_ref(v.view(T, hkv, dv), 1.0, eps)
        ok = slots >= 0
        k_cache.view(-1, hkv, dk)[slots[ok]] = k[ok].to(k_cache.dtype)
        v_cache.view(-1, hkv, dv)[slots[ok]] = v.view(T, hkv, dv)[ok].to(v_cache.dtype)
        return
    assert qkv.stride(1) == 1 and k_cache.dtype == qkv.dtype and (v_first is None or (v_first.stride(1) == 1 and v_first.dtype == qkv.dtype))
    rc = nat.lib().omni_qkv_prepare(
        nat.ptr(qkv), nat.c_int(qkv.stride(0)), nat.c_int(hq), nat.c_int(hkv), nat.c_int(dk), nat.c_int(dv), nat.ptr(q_w), nat.ptr(k_w),
        nat.c_float(eps), nat.ptr(cos_sin), nat.c_int(rot), nat.c_int(int(pairs)), nat.ptr(positions), nat.ptr(slots), nat.ptr(mix),
        nat.ptr(v_first if mix is not None else None), nat.c_int(v_first.stride(0) if mix is not None else 0), nat.c_int(int(v_norm)),
        nat.ptr(k_cache), nat.ptr(v_cache), nat.c_int(T), nat.c_int(_f32(qkv)), nat.stream())
    nat.check_rc(rc, "omni_qkv_prepare")


def latent_prepare(a, q_rank, kv0, kv_rank, rot, q_w, kv_w, eps, cos_sin, positions, slots, cache, latent_cols, q_cols, want_rows=False):
    """``a`` rows: q_rank columns of the query latent (0: there is none), and from column ``kv0`` on kv_rank of the key/value latent | rot
    of the shared key part.  The latents are normed, the key part rotated; latent | key part (``latent_cols`` and the rest of the cache's
    columns, zeros past the real sizes) are cached at ``slots``.  -> (query latent [T, q_cols] or None, the cached rows or None)."""
    T, D = a.shape[0], cache.shape[-1]
    if not a.is_cuda:
        cq = None
        if q_rank:
            cq = torch.zeros(T, q_cols, dtype=a.dtype)
            cq[:, :q_rank] = rms_ref(a[:, :q_rank].float(), q_w, eps).to(a.dtype)
        rows = torch.zeros(T, D, dtype=a.dtype)
        rows[:, :kv_rank] = rms_ref(a[:, kv0:kv0 + kv_rank].float(), kv_w, eps).to(a.dtype)
        kr = _rotate_half_ref(a[:, None, kv0 + kv_rank:kv0 + kv_rank + rot].float(), cos_sin, positions, rot)
        rows[:, latent_cols:latent_cols + rot] = kr[:, 0].to(a.dtype)
        ok = slots >= 0
        cache.view(-1, D)[slots[ok]] = rows[ok]
        return cq, rows if want_rows else None
    assert a.stride(1) == 1 and cache.is_contiguous() and cache.dtype == a.dtype
    cq = torch.empty(T, q_cols, dtype=a.dtype, device=a.device) if q_rank else None
    rows = torch.empty(T, D, dtype=a.dtype, device=a.device) if want_rows else None
    rc = nat.lib().omni_latent_prepare(
        nat.ptr(a), nat.c_int(a.stride(0)), nat.c_int(q_rank), nat.c_int(kv0), nat.c_int(kv_rank), nat.c_int(rot), nat.ptr(q_w),
        nat.ptr(kv_w), nat.c_float(eps), nat.ptr(cos_sin), nat.ptr(positions), nat.ptr(slots), nat.ptr(cq), nat.c_int(q_cols),
        nat.ptr(cache), nat.ptr(rows), nat.c_int(latent_cols), nat.c_int(D - latent_cols), nat.c_int(T), nat.c_int(_f32(a)), nat.stream())
    nat.check_rc(rc, "omni_latent_prepare")
    return cq, rows


def rotate_heads(x, rot, cos_sin, positions, out):
    """x [T, H, >= rot] (a column slice of every head) with its first ``rot`` entries rotated (halves) into ``out`` [T, H, cols], zeros
    past ``rot``.  ``out`` may be ``x``."""
    T, H, cols = out.shape
    if not x.is_cuda:
        y = _rotate_half_ref(x[..., :rot].float(), cos_sin, positions, rot).to(out.dtype)
        out[..., :rot] = y
        out[..., rot:] = 0
        return out
    assert x.dtype == out.dtype and x.stride(2) == 1 and out.stride(2) == 1
    rc = nat.lib().omni_rotate_heads(
        nat.ptr(x), nat.c_int64(x.stride(0)), nat.c_int(x.stride(1)), nat.c_int(T), nat.c_int(H), nat.c_int(rot), nat.ptr(cos_sin),
        nat.ptr(positions), nat.ptr(out), nat.c_int64(out.stride(0)), nat.c_int(out.stride(1)), nat.c_int(cols), nat.c_int(_f32(x)),
        nat.stream())
    nat.check_rc(rc, "omni_rotate_heads")
    return out


def gather_pages(cache, block_table, requests, pos0, first, end, total, longest):
    """Rows ``first[b]:end[b]`` of the result are the cached rows of request ``requests[b]`` from position ``pos0[b]`` on."""
    bs, D = cache.shape[1], cache.shape[2]
    if not cache.is_cuda:
        out, flat = torch.zeros(total, D, dtype=cache.dtype), cache.view(-1, D)
        for r, p, a, e in zip(requests.tolist(), pos0.tolist(), first.tolist(), end.tolist()):
            pos = torch.arange(p, p + e - a)
            out[a:e] = flat[block_table[r, pos // bs].long() * bs + pos % bs]
        return out
    assert cache.is_contiguous() and block_table.stride(1) == 1
    out = torch.empty(total, D, dtype=cache.dtype, device=cache.device)
    rc = nat.lib().omni_gather_pages(
        nat.ptr(cache), nat.c_int(D * cache.element_size()), nat.ptr(block_table), nat.c_int(block_table.stride(0)), nat.c_int(bs),
        nat.ptr(requests), nat.ptr(pos0), nat.ptr(first), nat.ptr(end), nat.c_int(requests.shape[0]), nat.c_int(longest), nat.ptr(out),
        nat.stream())
    nat.check_rc(rc, "omni_gather_pages")
    return out


def latent_attention(q, cache, latent_cols, *, positions, q_to_seq, slots, block_table, seq_lens, scale, window=0, gate=None, max_seq_len=0,
                     sink=None):
    """Attention in latent space: q [T, H, D] (latent part | rotated part) against the cached rows [blocks, block, D] that the rows'
    requests (``q_to_seq``) hold, row t seeing the last ``window`` of its first ``seq_lens[t]``; values are the first ``latent_cols``
    of the rows.  ``gate`` [T, H], ``sink`` [H]: as in :func:`paged_attention`.  -> [T, H, latent_cols]."""
    T, H, D = q.shape
    if q.is_cuda and q.dtype == torch.bfloat16 and (D, latent_cols) == (576, 512) and H <= 128 and (cache.shape[1] == 32 or cache.shape[1] % 64 == 0):
        from .attention import mla_decode
        return mla_decode(q, cache, block_table, seq_lens, scale, q_to_seq=q_to_seq, max_seq_len=max_seq_len, exact=True, window=window,
                          gate=gate, sink=sink)
    kv = cache.unsqueeze(2)
    out = paged_attention(q, kv, kv[..., :latent_cols], positions=positions, q_to_seq=q_to_seq, slots=slots, block_table=block_table,
                          seq_lens=seq_lens, scale=scale, window=window, gate=gate, max_seq_len=max_seq_len, rows_share=True, sink=sink)
    return out.view(T, H, latent_cols)


def latent_prefill_fits(dtype, d1, d2, dv, scale) -> bool:
    """Does the tensor-core kernel for portions of prompts take these head sizes and this (positive) scale?"""
    return scale > 0 and dtype == torch.bfloat16 and (d1 + 63) // 64 + (d2 + 63) // 64 <= 3 and dv <= 128


def latent_prefill(q, kv, k2, *, d1, dv, q_start, q_end, k_start, k_end, max_q, scale, window=0, gate=None, sink=None, out=None):
    """Attention over projected keys: q [T, H, d1 + d2], ``kv`` [K, H (d1 + dv)] = per head keys | values, ``k2`` [K, d2] key columns
    of all heads.  Request b has query rows q_start[b]:q_end[b] and key rows k_start[b]:k_end[b], whose last ones are its queries'.
    Writes those rows of ``out`` [T, H dv]."""
    T, H, d = q.shape
    d2 = d - d1
    assert q.is_cuda and q.dtype == kv.dtype == k2.dtype == torch.bfloat16 and q.stride(2) == 1 and q.stride(1) == d
    if out is None:
        out = torch.empty(T, H * dv, dtype=q.dtype, device=q.device)
    rc = nat.lib().omni_fmha_latent(
        nat.ptr(q), nat.c_int64(T), nat.c_int(q.stride(0)), nat.ptr(kv), nat.c_int64(kv.shape[0]), nat.c_int(kv.stride(0)), nat.ptr(k2),
        nat.c_int(k2.stride(0)), nat.ptr(q_start), nat.ptr(q_end), nat.ptr(k_start), nat.ptr(k_end), nat.c_int(q_start.shape[0]),
        nat.c_int(max_q), nat.c_int(H), nat.c_int(d1), nat.c_int(d2), nat.c_int(dv), nat.c_int(window), nat.c_float(scale),
        nat.ptr(gate), nat.c_int(gate.stride(0) if gate is not None else 0), nat.ptr(sink), nat.ptr(out), nat.c_int(out.stride(0)),
        nat.ptr(nat.status_buffer(q.device)), nat.stream())
    nat.check_rc(rc, "omni_fmha_latent")
    return out

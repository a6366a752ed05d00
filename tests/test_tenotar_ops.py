"""Every op that the Tenotar design adds, alone, against the plain implementation: CPU references and CUDA kernels, fp32 and bf16,
sizes on and off the tensor-core paths, keys just inside and just outside every mask, slots that hold another request's leftovers."""
import math

import pytest
import torch

import tenotar_oracle as oracle
from omni_infer_b200 import ops
from omni_infer_b200.layers.common import GeGLUMLP
from omni_infer_b200.layers.moe import ExpertMixture
from omni_infer_b200.models.config import ExpertsSpec
from omni_infer_b200.ops import attn_prepare as ap
from omni_infer_b200.ops import layer_list as ll
from omni_infer_b200.ops.streams import ExpertSum
from test_layer_list_ops import BF16, F32, RUNS, TOL, acts, batch_md, close, paged_case, rnd, run_portions


@pytest.fixture(autouse=True)
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


# ----------------------------------------------------------------------------- residual
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H", [(1, 8), (5, 37), (3, 200), (2, 4104), (4, 2050)])
@pytest.mark.parametrize("ones", [False, True])
def test_residual_with_the_norm_ahead(device, dtype, T, H, ones):
    ld, eps, w, b = ll.pad8(H + int(ones)), 1e-3, 1 + 0.2 * rnd(H, seed=2), rnd(H, seed=3, scale=0.1)
    x0 = torch.zeros(T, ll.pad8(H))
    x0[:, :H] = rnd(T, H, seed=1, scale=0.05)
    y, yd = acts(rnd(T, H, seed=4, scale=0.05), dtype, device, ll.pad8(H) + 8)
    for bias, scale in ((None, 1.0), (b, 0.3)):
        want = x0[:, :H].double() + yd + (0 if bias is None else bias.double())
        x = x0.clone().to(device)
        h = ll.add_norm(x, y, w.to(device), eps, dtype, ld=ld, ones=ones, bias=None if bias is None else bias.to(device), scale=scale)
        close(x[:, :H], want, 2e-6)
        close(h[:, :H], oracle.rms(want, eps) * w.double() * scale, TOL[dtype])
        assert h.dtype == dtype and h.shape == (T, ld) and not h[:, H + int(ones):].any() and (not ones or (h[:, H] == 1).all())
    table, td = acts(rnd(11, H, seed=7), dtype, device, ll.pad8(H))
    ids = torch.tensor([7, 0, 10, 3, 7][:T], device=device)
    x, h = ll.embed_norm(ids, table, w.to(device), eps, ld=ld, ones=ones)
    assert torch.equal(x[:, :H].double().cpu(), td[ids.cpu()])
    close(h[:, :H], oracle.rms(td[ids.cpu()], eps) * w.double(), TOL[dtype])
    assert not ones or (h[:, H] == 1).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("with_shared", [False, True])
def test_expert_parts_are_summed_into_the_residual(device, dtype, with_shared):
    T, H, k = 6, 40, 3
    y, yd = acts(rnd(20, H, seed=1), dtype, device)
    sh, sd = acts(rnd(T, H, seed=2), dtype, device)
    row_of = torch.randperm(20, generator=torch.Generator().manual_seed(1))[:T * k].int()
    row_of[7], row_of[12:15] = -1, -1
    parts = ExpertSum(y, row_of.to(device), torch.zeros(T, k, dtype=torch.int32, device=device), torch.zeros(T, k, device=device), 9, None,
                      sh if with_shared else None)
    if device == "cpu":
        parts.h = torch.zeros(T, H)
    want = rnd(T, H, seed=3).double()
    x = want.float().to(device)
    for t in range(T):
        want[t] += sum(yd[r] for r in row_of.view(T, k)[t].tolist() if r >= 0) + (sd[t] if with_shared else 0)
    h = ll.add_norm(x, parts, torch.ones(H, device=device), 1e-5, dtype, ld=H)
    close(x, want, 2e-6)
    close(h, oracle.rms(want, 1e-5), TOL[dtype])


# ----------------------------------------------------------------------------- head norm, rotation, mixing, cache write
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv,rot", [(4, 2, 16, 24, 16), (3, 1, 9, 5, 6), (2, 2, 8, 8, 0), (6, 3, 40, 32, 8), (1, 1, 136, 8, 64), (3, 3, 11, 7, 10),
                                          (2, 1, 300, 12, 20)])
@pytest.mark.parametrize("pairs,normed,mix", [(True, True, True), (False, True, False), (True, False, False), (False, False, True)])
def test_heads_prepared(device, dtype, H, G, d, dv, rot, pairs, normed, mix):
    T, eps, bs, nb = 7, 1e-3, 16, 5
    nq, nk, nv = H * d, G * d, G * dv
    qkv, ref = acts(rnd(T, nq + nk + nv, seed=1, scale=0.1), dtype, device, ll.pad8(nq + nk + nv))
    first, fd = acts(rnd(T, nv, seed=5), dtype, device, ll.pad8(nv) + 4)
    qw, kw, lam = 1 + 0.3 * rnd(d, seed=2), 1 + 0.3 * rnd(d, seed=3), torch.tensor([0.3])
    pos, slots = torch.tensor([0, 1, 2, 300, 301, 17, 900]), torch.tensor([3, 70, 11, -1, 0, 79, 33])
    cs = ops.rope_cos_sin_table(rot, 1024, 500.0).to(device) if rot else None
    kc = torch.full((nb, bs, G, d), 7.0, dtype=dtype, device=device)
    vc = torch.full((nb, bs, G, dv), 7.0, dtype=dtype, device=device)
    ap.qkv_prepare(qkv, H, G, d, dv, qw.to(device) if normed else None, kw.to(device) if normed else None, eps, cs, rot, pairs, pos.to(device),
                   slots.to(device), kc, vc, mix=lam.to(device) if mix else None, v_first=first[:, :nv] if mix else None)
    order = (oracle.neighbours if pairs else oracle.halves)(rot)

    def want(x, w, heads):
        x = x.reshape(T, heads, d)
        x = oracle.rms(x, eps) * w.double() if normed else x
        full = torch.zeros(901, heads, d, dtype=torch.double)
        full[pos] = x
        return oracle.rotate(full, {"base": 500.0, "dims": rot}, order)[pos] if rot else x

    close(qkv[:, :nq].reshape(T, H, d), want(ref[:, :nq], qw, H), TOL[dtype])
    ok = slots >= 0
    at = slots[ok].to(device)
    close(kc.view(-1, G, d)[at], want(ref[:, nq:nq + nk], kw, G)[ok], TOL[dtype])
    v = ref[:, nq + nk:]
    v = oracle.mix_values(v, fd, 0.3) if mix else v
    close(vc.view(-1, nv)[at], v[ok], TOL[dtype])
    assert torch.equal(qkv[:, nq:nq + nk + nv].double().cpu(), ref[:, nq:])      # the values themselves stay: others may mix them in
    rest = torch.ones(nb * bs, dtype=torch.bool)
    rest[slots[ok]] = False
    assert (kc.view(-1, G, d)[rest.to(device)] == 7).all() and (vc.view(-1, G, dv)[rest.to(device)] == 7).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("C,taps,sizes", [(16, 4, [2, 1, 3]), (40, 3, [17, 64, 2, 1, 1]), (13, 2, [400]), (24, 1, [5]), (9, 7, [2]), (520, 4, [1])])
def test_convolution_without_bias_and_activation(device, dtype, C, taps, sizes):
    lens, w = [40, 1, 23, 9], rnd(C, taps, seed=1)
    xs = [acts(rnd(n, C, seed=10 + r), dtype, device, ll.pad8(C) + 8) for r, n in enumerate(lens)]
    state = torch.full((6, taps - 1, C), 9.0, dtype=dtype, device=device)        # leftovers
    slots, got = [4, 0, 3, 1], [[] for _ in lens]

    def call(batch):
        md = batch_md(batch, slots, device)
        if all(m == 1 for _, _, m in batch):
            md["cu_q"] = None
        y = ll.short_conv(torch.cat([xs[r][0][a:a + m] for r, a, m in batch])[:, :C], w.t().contiguous().to(device), None, state, **md)
        at = 0
        for r, _, m in batch:
            got[r].append(y[at:at + m, :C])
            at += m

    run_portions(lens, sizes, call)
    for r in range(len(lens)):
        close(torch.cat(got[r]), oracle.short_conv(xs[r][1], w.double()), TOL[dtype])


# ----------------------------------------------------------------------------- masks and scores
def want_attention(lens, portions, ks, vs, qs, scale, mask, softcap=None, slopes=None):
    out = []
    for n, m, k, v, q in zip(lens, portions, ks, vs, qs):
        full = torch.zeros(n, *q.shape[1:], dtype=torch.double)
        full[n - m:] = q
        out.append(oracle.attend(full, k, v, scale, mask(n), softcap, slopes)[n - m:].reshape(m, -1))
    return torch.cat(out)


MASKS = [dict(window=37, keep_first=5), dict(window=64, keep_first=64), dict(window=1, keep_first=1), dict(window=65, keep_first=130),
         dict(window=20, keep_first=1000), dict(chunk=64), dict(chunk=100), dict(chunk=1), dict(chunk=500), dict()]
SHAPES = [(4, 2, 64, 64), (8, 2, 72, 104), (4, 4, 16, 24), (3, 1, 9, 5), (6, 2, 192, 40), (20, 1, 32, 32), (2, 2, 200, 136)]


def mask_of(m):
    return lambda n: oracle.chunk_mask(n, m["chunk"]) if m.get("chunk") else oracle.window_mask(n, m.get("window") or n + 1, m.get("keep_first", 0))


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv", SHAPES)
@pytest.mark.parametrize("modified", [False, True], ids=["plain", "capped"])
@pytest.mark.parametrize("mask", MASKS, ids=lambda m: "-".join(f"{k}{v}" for k, v in m.items()) or "all")
def test_masks(device, dtype, H, G, d, dv, modified, mask):
    """Portions, the same rows as single tokens, and the kernel for any shape."""
    if device == "cpu" and (H * d > 300 or not modified):
        pytest.skip("covered by the other sizes")
    scale, kw, ref = 1.7 / math.sqrt(d), dict(mask), ()
    if modified:
        kw.update(softcap=1.3, slopes=torch.tensor(oracle.slopes_of(H), dtype=F32, device=device))
        ref = (1.3, oracle.slopes_of(H))
    lens, portions = [5, 200, 64, 321, 130], [5, 130, 1, 2, 129]
    q, kc, vc, a, cu, ks, vs, qs = paged_case(lens, portions, H, G, d, dv, 64, dtype, device, seed=d)
    want = want_attention(lens, portions, ks, vs, qs, scale, mask_of(mask), *ref)
    for any_shape in (False, True) if device == "cuda" else (False,):
        got = ll.paged_attention(q, kc, vc, scale=scale, cu_q=cu, max_q=max(portions), max_seq_len=max(lens), any_shape=any_shape, **kw, **a)
        close(got[:, : H * dv], want, TOL[dtype])
    lens = [1, 63, 64, 65, 700, 33]
    q, kc, vc, a, _, ks, vs, qs = paged_case(lens, [1] * len(lens), H, G, d, dv, 16, dtype, device, seed=dv)
    a["slots"][1], a["seq_lens"][1] = -1, 0                       # a padding row
    want = want_attention(lens, [1] * len(lens), ks, vs, qs, scale, mask_of(mask), *ref)
    want[1] = 0
    close(ll.paged_attention(q, kc, vc, scale=scale, max_seq_len=max(lens), **kw, **a)[:, : H * dv], want, TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["portion", "decoded"])
@pytest.mark.parametrize("mask,at,seen", [
    (dict(window=100, keep_first=6), 160, True), (dict(window=100, keep_first=6), 159, False), (dict(window=100, keep_first=6), 5, True),
    (dict(window=100, keep_first=6), 6, False), (dict(window=64, keep_first=65), 64, True), (dict(window=64, keep_first=65), 65, False),
    (dict(window=64, keep_first=1), 0, True), (dict(window=64, keep_first=0), 0, False), (dict(chunk=200), 200, True),
    (dict(chunk=200), 199, False), (dict(chunk=64), 256, True), (dict(chunk=64), 255, False), (dict(chunk=259), 259, True)])
def test_edges_of_the_masks(device, dtype, decode, mask, at, seen):
    """A key that dominates every score of the last query sits just inside or just outside."""
    H, G, d, dv, n = 2, 1, 64, 64, 260
    i, m = n - 1, 1 if decode else 3
    q, kc, vc, a, cu, ks, vs, qs = paged_case([n], [m], H, G, d, dv, 64, dtype, device, spike=[(0, i, at, 3.0)])
    got = ll.paged_attention(q, kc, vc, scale=1 / math.sqrt(d), cu_q=None if decode else cu, max_q=m, max_seq_len=n, **mask, **a)
    close(got, want_attention([n], [m], ks, vs, qs, 1 / math.sqrt(d), mask_of(mask)), TOL[dtype])
    v = vs[0][at, 0].repeat(H)
    assert (float((got[-1].double().cpu() - v).norm() / v.norm()) < 0.2) == (seen or at == i)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["portion", "decoded"])
def test_cap_and_distance_change_what_wins(device, dtype, decode):
    """A far key with a huge score: wins as it is, loses to nearer ones once it is capped and its distance counts - by head."""
    H, d, n, m = 8, 64, 300, 1 if decode else 5
    q, kc, vc, a, cu, ks, vs, qs = paged_case([n], [m], H, 1, d, 64, 64, dtype, device, spike=[(0, n - 1, 40, 60.0)])
    kw = dict(scale=0.05, cu_q=None if decode else cu, max_q=m, max_seq_len=n)
    slopes = oracle.slopes_of(H)
    for ref, opts in (((), {}), ((8.0, None), dict(softcap=8.0)), ((None, slopes), dict(slopes=torch.tensor(slopes, device=device))),
                      ((8.0, slopes), dict(softcap=8.0, slopes=torch.tensor(slopes, device=device)))):
        got = ll.paged_attention(q, kc, vc, **kw, **opts, **a)
        close(got, want_attention([n], [m], ks, vs, qs, 0.05, mask_of({}), *ref), TOL[dtype])
    far = vs[0][40, 0]
    share = [float(got[-1].view(H, 64)[h].double().cpu() @ far / far.norm() ** 2) for h in (0, H - 1)]
    assert abs(share[0]) < 0.3 and share[1] > 0.6, share      # the steepest head does not see it, the flattest one does


# ----------------------------------------------------------------------------- latents
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("qr,kr,rot,C,R", [(24, 40, 8, 40, 8), (5, 13, 6, 16, 8), (96, 260, 16, 512, 64), (768, 512, 64, 512, 64), (3, 3, 2, 8, 8)])
def test_latents_prepared(device, dtype, qr, kr, rot, C, R):
    T, eps, bs, nb, kv0 = 6, 1e-3, 16, 4, ll.pad8(qr)
    raw = torch.zeros(T, kv0 + kr + rot + 3)
    raw[:, :qr], raw[:, kv0:] = rnd(T, qr, seed=1, scale=0.1), rnd(T, kr + rot + 3, seed=2, scale=0.1)
    a, ref = acts(raw, dtype, device, ll.pad8(raw.shape[1]))
    qw, cw, pos, slots = 1 + 0.2 * rnd(qr, seed=3), 1 + 0.2 * rnd(kr, seed=4), torch.tensor([0, 1, 2, 77, 78, 500]), torch.tensor([5, 6, 7, -1, 63, 0])
    cache = torch.full((nb, bs, C + R), 7.0, dtype=dtype, device=device)
    cs = ops.rope_cos_sin_table(rot, 512, 300.0).to(device)
    cq, rows = ap.latent_prepare(a, qr, kv0, kr, rot, qw.to(device), cw.to(device), eps, cs, pos.to(device), slots.to(device), cache, C, kv0, True)
    close(cq[:, :qr], oracle.rms(ref[:, :qr], eps) * qw.double(), TOL[dtype])
    want = torch.zeros(T, C + R, dtype=torch.double)
    want[:, :kr] = oracle.rms(ref[:, kv0:kv0 + kr], eps) * cw.double()
    full = torch.zeros(501, 1, rot, dtype=torch.double)
    full[pos, 0] = ref[:, kv0 + kr:kv0 + kr + rot]
    want[:, C:C + rot] = oracle.rotate(full, {"base": 300.0, "dims": rot}, oracle.halves(rot))[pos, 0]
    close(rows, want, TOL[dtype])
    assert not cq[:, qr:].any() and not rows[:, kr:C].any() and not rows[:, C + rot:].any()
    ok = slots >= 0
    assert torch.equal(cache.view(-1, C + R)[slots[ok].to(device)], rows[ok.to(device)])
    assert int((cache == 7).all(-1).sum()) == nb * bs - int(ok.sum())
    # the same part of a head elsewhere and in place
    x, xd = acts(rnd(T, 3 * (rot + 10), seed=6), dtype, device)
    x = x.view(T, 3, rot + 10)[..., 4 if rot % 4 == 0 else 3:]
    part = xd.view(T, 3, rot + 10)[..., 4 if rot % 4 == 0 else 3:][..., :rot]
    full = torch.zeros(501, 3, rot, dtype=torch.double)
    full[pos] = part
    want = oracle.rotate(full, {"base": 300.0, "dims": rot}, oracle.halves(rot))[pos]
    out = torch.full((T, 3, C + R), 7.0, dtype=dtype, device=device)
    ap.rotate_heads(x, rot, cs, pos.to(device), out[..., C:])
    close(out[..., C:C + rot], want, TOL[dtype])
    assert (out[..., :C] == 7).all() and not out[..., C + rot:].any()
    ap.rotate_heads(x, rot, cs, pos.to(device), x[..., :rot])
    close(x[..., :rot], want, TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
def test_gathered_pages(device, dtype):
    cache = rnd(9, 16, 24, seed=1).to(dtype).to(device)
    bt = torch.tensor([[3, 8, 1, 0], [5, 2, 7, 6]], dtype=torch.int32, device=device)
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=device)      # noqa: E731
    out = ap.gather_pages(cache, bt, i32(1, 0, 1), i32(15, 0, 63), i32(0, 20, 53), i32(20, 53, 54), 54, 33)
    flat = cache.view(-1, 24)
    rows = [(5, 2, 7, 6)[p // 16] * 16 + p % 16 for p in range(15, 35)] + [(3, 8, 1)[p // 16] * 16 + p % 16 for p in range(33)] + [6 * 16 + 15]
    assert torch.equal(out, flat[torch.tensor(rows, device=device)])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,C,R", [(4, 64, 16), (20, 96, 32), (3, 16, 8), (16, 512, 64), (5, 512, 64), (2, 200, 56), (3, 296, 24), (100, 512, 64), (2, 600, 8)])
@pytest.mark.parametrize("window", [0, 1, 37, 64, 65, 200])
def test_attention_in_latent_space(device, dtype, H, C, R, window):
    """Rows that stand alone, and several rows of a request; values are a part of the keys; a gate per row and head."""
    if device == "cpu" and (H > 4 or window in (64, 65)):
        pytest.skip("covered by the other sizes")
    lens, portions, bs = [1, 65, 700, 130, 64], [1, 1, 2, 3, 1], 64
    q, kc, _, a, cu, ks, _, qs = paged_case(lens, portions, H, 1, C + R, 8, bs, dtype, device, seed=C + window)
    T = q.shape[0]
    gate, gd = acts(rnd(T, H + 3, seed=9), dtype, device)
    a["seq_lens"] = (a["positions"] + 1).int()
    scale = 1.5 / math.sqrt(C + R)
    got = ap.latent_attention(q.contiguous(), kc.squeeze(2), C, scale=scale, window=window, gate=gate[:, :H], max_seq_len=max(lens), **a)
    want = want_attention(lens, portions, ks, [k[..., :C] for k in ks], qs, scale, mask_of(dict(window=window)))
    want = want.view(T, H, C) * oracle.sigmoid(gd[:, :H])[:, :, None]
    close(got, want, TOL[dtype])


@pytest.mark.gpu
@pytest.mark.parametrize("H,d1,d2,dv", [(4, 128, 64, 128), (3, 40, 16, 88), (2, 8, 8, 8), (5, 64, 64, 72), (2, 104, 40, 128), (1, 72, 24, 16)])
@pytest.mark.parametrize("window", [0, 1, 70, 64, 129])
def test_attention_over_projected_keys(H, d1, d2, dv, window):
    """Requests anywhere in the rows, some of the step's rows left out, keys of which only the last belong to queries."""
    portions, ctx = [130, 20, 300, 9], [0, 200, 69, 1]
    lens = [c + n for c, n in zip(ctx, portions)]
    T, K = sum(portions) + 7, sum(lens) + 5
    q, qd = acts(rnd(T, H * (d1 + d2), seed=1), BF16, "cuda")
    kv, kd = acts(rnd(K, H * (d1 + dv), seed=2), BF16, "cuda")
    k2, k2d = acts(rnd(K, d2, seed=3), BF16, "cuda", d2 + 16)
    gate, gd = acts(rnd(T, H, seed=4), BF16, "cuda", H + 5)
    q0, k0 = [3, 133, 155, 455], [4, 134, 354, 723]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")      # noqa: E731
    out = torch.full((T, H * dv), 5.0, dtype=BF16, device="cuda")
    ap.latent_prefill(q.view(T, H, d1 + d2), kv, k2[:, :d2], d1=d1, dv=dv, q_start=i32(q0), q_end=i32([a + n for a, n in zip(q0, portions)]),
                      k_start=i32(k0), k_end=i32([a + n for a, n in zip(k0, lens)]), max_q=300, scale=1.6 / math.sqrt(d1 + d2), window=window,
                      gate=gate[:, :H], out=out)
    rest = torch.ones(T, dtype=torch.bool)
    for a, n, b, m in zip(q0, portions, k0, lens):
        rows = kd[b:b + m].view(m, H, d1 + dv)
        k = torch.cat([rows[..., :d1], k2d[b:b + m, None].expand(m, H, d2)], -1)
        full = torch.zeros(m, H, d1 + d2, dtype=torch.double)
        full[m - n:] = qd[a:a + n].view(n, H, d1 + d2)
        want = oracle.attend(full, k, rows[..., d1:], 1.6 / math.sqrt(d1 + d2), mask_of(dict(window=window))(m))[m - n:]
        close(out[a:a + n].view(n, H, dv), want * oracle.sigmoid(gd[a:a + n])[:, :, None], TOL[BF16])
        rest[a:a + n] = False
    assert (out[rest.cuda()] == 5).all()


# ----------------------------------------------------------------------------- feed-forward
def put(layer, w, prefix):
    for name, (p, r0, rows, cols) in layer.checkpoint_targets().items():
        (p.data[r0:r0 + rows] if cols is None else p.data[r0:r0 + rows, :cols]).copy_(w[prefix + name])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H,ff,sff,E,top", [(1, 16, 8, 16, 3, 2), (70, 64, 128, 256, 8, 3), (9, 37, 13, 21, 5, 5), (150, 72, 24, 0, 6, 1), (300, 64, 128, 40, 9, 4)])
def test_expert_mixture(device, dtype, T, H, ff, sff, E, top):
    m = {"router": {"experts": E, "top": top}, "expert": {"ff": ff}, "shared": {"ff": sff} if sff else None}
    w = {"p.router": rnd(E, H, seed=1, scale=1.5 / math.sqrt(H)).to(dtype), "p.router.b": rnd(E, seed=2)}
    for i, (e, n) in enumerate([(f"e{e}.", ff) for e in range(E)] + ([("shared.", sff)] if sff else [])):
        for j, (c, o, k) in enumerate((("gate", n, H), ("up", n, H), ("down", H, n))):
            w[f"p.{e}{c}"] = rnd(o, k, seed=10 + 3 * i + j, scale=1.5 / math.sqrt(k)).to(dtype)
    layer = ExpertMixture(ExpertsSpec(E, top, ff, shared_ff=sff, act="swiglu", weighting="chosen"), H, dtype=dtype, device=device)
    put(layer, w, "p.")
    x, xd = acts(rnd(T, H, seed=4), dtype, device, ll.pad8(H))
    wd = {k: v.double() for k, v in w.items()}
    order = oracle.linear(xd, wd, "p.router").sort(-1, descending=True).values
    clear = torch.ones(T, dtype=torch.bool) if top == E else (order[:, top - 1] - order[:, top]) > 2e-2      # no close choice
    assert clear.float().mean() > 0.8
    close(layer(x).total()[clear.to(device), :H], oracle.mixture(xd, wd, "p.", m)[clear], TOL[dtype] * 2)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_router_bias_moves_choice_and_weights(device, dtype):
    z, b = torch.tensor([[1.0, 0.5, 0.0, -3.0]], device=device), torch.tensor([-2.0, 0.0, 0.0, 4.0], device=device)
    ids, w = ops.router_topk(z, 2, renorm=True, logit_bias=b)
    assert ids.tolist() == [[3, 1]]
    assert w[0].tolist() == pytest.approx(torch.softmax(torch.tensor([1.0, 0.5]), 0).tolist(), rel=1e-6)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,K,I", [(1, 16, 8), (70, 64, 128), (9, 37, 13), (130, 71, 256), (33, 24, 136)])
def test_feed_forward_with_biases(device, dtype, T, K, I):
    m = GeGLUMLP(K, I, dtype=dtype, device=device, epi="swiglu", bias=True)
    w = {f"m.{c}": rnd(o, k, seed=i, scale=1.5 / math.sqrt(k)).to(dtype) for i, (c, o, k) in enumerate((("gate", I, K), ("up", I, K), ("down", K, I)))}
    w.update({f"m.{c}.b": rnd(o, seed=7 + i).to(dtype) for i, (c, o) in enumerate((("gate", I), ("up", I), ("down", K)))})
    m.zero_padding()
    put(m, w, "m.")
    x, xd = acts(rnd(T, K, seed=4), dtype, device, m.in_cols)
    x[:, K] = 1
    got = m(x)[:, :K].double().cpu() + m.out_bias.double().cpu()
    close(got, oracle.gated(xd, {k: v.double() for k, v in w.items()}, "m."), TOL[dtype] * 2)

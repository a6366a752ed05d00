"""Every op that the Zusotar design adds, alone, against the plain implementation: CPU references and CUDA kernels, fp32 and bf16,
sizes on and off the tensor-core paths, keys just inside and just outside every window, slots that hold another request's leftovers."""
import math

import pytest
import torch

import zusotar_oracle as oracle
from omni_infer_b200 import ops
from omni_infer_b200.layers.latent_attention import LatentAttention
from omni_infer_b200.layers.moe import ExpertMixture
from omni_infer_b200.models.config import ExpertsSpec, LatentSpec
from omni_infer_b200.ops import attn_prepare as ap
from omni_infer_b200.ops import depth
from omni_infer_b200.ops import layer_list as ll
from omni_infer_b200.ops import matrix_state as ms
from omni_infer_b200.ops.streams import ExpertSum
from test_fimudra_ops import CUTS, by_cuts
from test_layer_list_ops import BF16, F32, RUNS, TOL, acts, close, paged_case, rnd


@pytest.fixture(autouse=True)
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def padded(x, ld, device):
    out = torch.full((*x.shape[:-1], ld), 7.0, device=device)
    out[..., :x.shape[-1]] = x.to(device)
    return out


# ----------------------------------------------------------------------------- embedding, connection of the layers
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H", [(1, 8), (5, 37), (3, 200), (2, 4104), (4, 2050)])
def test_embedding_with_positions(device, dtype, T, H):
    ld, eps, w = ll.pad8(H), 1e-3, 1 + 0.2 * rnd(H, seed=2)
    table, td = acts(rnd(11, H, seed=7, scale=0.05), dtype, device, ld)
    pos, pd = acts(rnd(9, H, seed=8, scale=0.05), dtype, device, ld + 8)
    ids, at = torch.tensor([7, 0, 10, 3, 7][:T]), torch.tensor([8, 0, 3, 9, 2][:T])      # position 9 is past the table
    for where in (pos, None):
        want = td[ids].clone()
        if where is not None:
            want += torch.where(at[:, None] < 9, pd[at.clamp_max(8)], 0.0)
        x = torch.empty(T, ld, device=device)
        h = depth.embed_positions(ids.to(device), table, at.to(device), where, x, w.to(device), eps, ld=ld + 8)
        close(x[:, :H], want, 1e-6)
        close(h[:, :H], oracle.rms(want, eps) * w.double(), TOL[dtype])
        assert h.dtype == dtype and h.shape == (T, ld + 8) and not h[:, H:].any()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H", [(1, 8), (5, 37), (3, 200), (2, 4104), (4, 2050), (2, 9000)])
def test_norm_behind_the_average_and_the_norm_ahead(device, dtype, T, H):
    ld, eps, mult = ll.pad8(H), 1e-3, 0.35
    wb, wn = 1 + 0.2 * rnd(H, seed=1), 1 + 0.2 * rnd(H, seed=2)
    x0, past = rnd(T, H, seed=3), rnd(4, T, H, seed=4)
    y, yd = acts(rnd(T, H, seed=5, scale=0.05), dtype, device, ld + 8)      # small outputs: eps counts
    summed = x0.double() + mult * oracle.rms(yd, eps) * wb.double()
    dev = lambda t: t.to(device)        # noqa: E731
    # between the sublayers of a layer; in place and elsewhere
    src = padded(x0, ld, device)
    dst = torch.full_like(src, 3.0)
    for out in (dst, src):
        h = depth.both_norms_step(src, out, y, dev(wb), mult, dev(wn), eps, dtype, ld=ld + 16)
        close(out[:, :H], summed, 2e-6)
        close(h[:, :H], oracle.rms(summed, eps) * wn.double(), TOL[dtype])
        assert h.dtype == dtype and h.shape == (T, ld + 16) and not h[:, H:].any()
    # behind layer n - 1, with room for its result and without (the last layer)
    for n, room in ((1, 4), (3, 4), (4, 4)):
        a = rnd(n + 1, seed=6 + n)
        results = padded(past[:room], ld, device)
        src = padded(x0, ld, device)
        h = depth.both_norms_step(src, src, y, dev(wb), mult, dev(wn), eps, dtype, ld=ld, results=results, average=dev(a))
        want = oracle.depth_average(a.double(), [*past[:n].double(), summed])
        close(src[:, :H], want, 2e-6)
        close(h[:, :H], oracle.rms(want, eps) * wn.double(), TOL[dtype])
        kept = past[:room].double().clone()
        if n < room:
            kept[n] = summed
        close(results[..., :H], kept, 2e-6)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("with_shared", [False, True])
def test_expert_parts_pass_through_the_norm_behind(device, dtype, with_shared):
    T, H, k = 6, 40, 3
    y, yd = acts(rnd(20, H, seed=1), dtype, device)
    sh, sd = acts(rnd(T, H, seed=2), dtype, device)
    row_of = torch.randperm(20, generator=torch.Generator().manual_seed(1))[:T * k].int()
    row_of[7], row_of[12:14] = -1, -1
    parts = ExpertSum(y, row_of.to(device), torch.zeros(T, k, dtype=torch.int32, device=device), torch.zeros(T, k, device=device), 9,
                      torch.zeros(T, H, device=device), sh if with_shared else None)
    total = torch.zeros(T, H, dtype=torch.double)
    for t in range(T):
        total[t] = sum(yd[r] for r in row_of.view(T, k)[t].tolist() if r >= 0) + (sd[t] if with_shared else 0)
    x0, one = rnd(T, H, seed=3), torch.ones(H, device=device)
    x = x0.clone().to(device)
    h = depth.both_norms_step(x, x, parts, one, 0.7, one, 1e-5, dtype, ld=H)
    want = x0.double() + 0.7 * oracle.rms(total, 1e-5)
    close(x, want, 2e-6)
    close(h, oracle.rms(want, 1e-5), TOL[dtype])


# ----------------------------------------------------------------------------- normed values
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 24), (3, 1, 9, 5), (6, 3, 40, 32), (1, 1, 136, 8), (2, 1, 12, 300), (12, 12, 8, 1)])
def test_values_are_normed_on_their_way_to_the_cache(device, dtype, H, G, d, dv):
    T, eps, bs, nb = 7, 1e-3, 16, 5
    nq, nk, nv = H * d, G * d, G * dv
    qkv, ref = acts(rnd(T, nq + nk + nv, seed=1, scale=0.05), dtype, device, ll.pad8(nq + nk + nv) + 8)
    slots = torch.tensor([3, 70, 11, -1, 0, 79, 33])
    kc = torch.full((nb, bs, G, d), 7.0, dtype=dtype, device=device)
    vc = torch.full((nb, bs, G, dv), 7.0, dtype=dtype, device=device)
    ap.qkv_prepare(qkv, H, G, d, dv, None, None, eps, None, 0, False, torch.arange(T, device=device), slots.to(device), kc, vc, v_norm=True)
    ok = slots >= 0
    at = slots[ok].to(device)
    close(vc.view(-1, G, dv)[at], oracle.rms(ref[:, nq + nk:].view(T, G, dv), eps)[ok], TOL[dtype])
    assert torch.equal(kc.view(-1, nk)[at].double().cpu(), ref[ok, nq:nq + nk])
    assert torch.equal(qkv[:, :nq + nk + nv].double().cpu(), ref)
    rest = torch.ones(nb * bs, dtype=torch.bool)
    rest[slots[ok]] = False
    assert (kc.view(-1, G, d)[rest.to(device)] == 7).all() and (vc.view(-1, G, dv)[rest.to(device)] == 7).all()


# ----------------------------------------------------------------------------- windows, distance bias, gates
def want_attention(lens, portions, ks, vs, qs, scale, size, r=None, sink=None):
    out = []
    for n, m, k, v, q in zip(lens, portions, ks, vs, qs):
        full = torch.zeros(n, *q.shape[1:], dtype=torch.double)
        full[n - m:] = q
        rep = q.shape[1] // k.shape[1]
        s = torch.einsum("ihd,jhd->hij", full, k.repeat_interleave(rep, 1)) * scale
        if r is not None:
            s = s - oracle.distance_bias(n, r[0].double(), r[1].double())
        mask = oracle.window_mask(n, size) if size else oracle.causal_mask(n)
        out.append(oracle.softmax_values(s, mask, v.repeat_interleave(rep, 1), sink)[n - m:].reshape(m, -1))
    return torch.cat(out)


SHAPES = [(4, 2, 64, 64), (8, 2, 72, 104), (4, 4, 16, 24), (3, 1, 9, 5), (6, 2, 192, 40), (20, 1, 32, 32), (2, 2, 200, 136)]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv", SHAPES)
@pytest.mark.parametrize("size", [0, 1, 37, 64, 65, 129, 500])
def test_logarithmic_bias_and_gates(device, dtype, H, G, d, dv, size):
    """Portions, the same rows as single tokens, and the kernel for any shape."""
    if device == "cpu" and (H * d > 300 or size in (64, 129)):
        pytest.skip("covered by the other sizes")
    scale, r = 1.7 / math.sqrt(d), (rnd(H, seed=3) * 1.5, torch.exp(rnd(H, seed=4) * 2 - 1))      # either sign of r1
    kw = dict(scale=scale, window=size, log_bias=tuple(t.to(device) for t in r))
    for lens, portions, bs in (([5, 200, 64, 321, 130], [5, 130, 1, 2, 129], 64), ([1, 63, 64, 65, 700, 33], [1] * 6, 16)):
        decode = portions[0] == 1
        q, kc, vc, a, cu, ks, vs, qs = paged_case(lens, portions, H, G, d, dv, bs, dtype, device, seed=d + size)
        T = q.shape[0]
        gate, gd = acts(rnd(T, H * dv, seed=9), dtype, device, ll.pad8(H * dv) + 8)
        want = want_attention(lens, portions, ks, vs, qs, scale, size, r)
        if decode:
            a["slots"][1], a["seq_lens"][1] = -1, 0                       # a padding row
            want[1] = 0
        how = dict(cu_q=None if decode else cu, max_q=max(portions), max_seq_len=max(lens))
        for any_shape in (False, True) if device == "cuda" and not decode else (False,):
            close(ll.paged_attention(q, kc, vc, any_shape=any_shape, **how, **kw, **a)[:, :H * dv], want, TOL[dtype])
            got = ll.paged_attention(q, kc, vc, any_shape=any_shape, gate=gate[:, :H * dv], **how, **kw, **a)[:, :H * dv]
            close(got, want * oracle.sigmoid(gd), TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["portion", "decoded"])
def test_the_distance_decides_by_head(device, dtype, decode):
    """A far key with the highest score: wins where the bias is flat, loses where it is steep, wins more where it is negative."""
    H, d, n, m = 4, 64, 300, 1 if decode else 5
    q, kc, vc, a, cu, ks, vs, qs = paged_case([n], [m], H, 1, d, 64, 64, dtype, device, spike=[(0, n - 1, 40, 30.0)])
    r = torch.tensor([0.0, 6.0, 6.0, -1.0]), torch.tensor([1.0, 1e-4, 2.0, 0.5])
    kw = dict(scale=0.05, cu_q=None if decode else cu, max_q=m, max_seq_len=n, log_bias=tuple(t.to(device) for t in r))
    got = ll.paged_attention(q, kc, vc, **kw, **a)
    close(got, want_attention([n], [m], ks, vs, qs, 0.05, 0, r), TOL[dtype])
    far = vs[0][40, 0]
    share = [float(got[-1].view(H, 64)[h].double().cpu() @ far / far.norm() ** 2) for h in range(H)]
    assert share[0] > 0.6 and share[1] > 0.6 and abs(share[2]) < 0.3 and share[3] > share[0] - 0.05, share


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["portion", "decoded"])
@pytest.mark.parametrize("size", [48, 64, 100, 129])
def test_window_edge_with_the_bias(device, dtype, decode, size):
    """A key that dominates every score of the last query sits just inside and just outside its window."""
    H, d, n, m = 2, 64, 260, 1 if decode else 3
    r = torch.tensor([0.3, 0.1]), torch.tensor([0.2, 1.0])
    for dist, seen in ((size - 1, True), (size, False)):
        q, kc, vc, a, cu, ks, vs, qs = paged_case([n], [m], H, 1, d, 64, 64, dtype, device, spike=[(0, n - 1, n - 1 - dist, 3.0)])
        got = ll.paged_attention(q, kc, vc, scale=1 / 8, window=size, cu_q=None if decode else cu, max_q=m, max_seq_len=n,
                                 log_bias=tuple(t.to(device) for t in r), **a)
        close(got, want_attention([n], [m], ks, vs, qs, 1 / 8, size, r), TOL[dtype])
        v = vs[0][n - 1 - dist, 0].repeat(H)
        assert (float((got[-1].double().cpu() - v).norm() / v.norm()) < 0.3) == seen


# ----------------------------------------------------------------------------- latents
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("kr,rot,C,R", [(40, 8, 40, 8), (13, 6, 16, 8), (260, 16, 512, 64), (512, 64, 512, 64), (3, 2, 8, 8)])
def test_latents_without_a_query_latent(device, dtype, kr, rot, C, R):
    T, eps, bs, nb, kv0 = 6, 1e-3, 16, 4, 24
    raw = rnd(T, kv0 + kr + rot + 3, seed=1, scale=0.05)
    a, ref = acts(raw, dtype, device, ll.pad8(raw.shape[1]))
    cw, pos, slots = 1 + 0.2 * rnd(kr, seed=4), torch.tensor([0, 1, 2, 77, 78, 500]), torch.tensor([5, 6, 7, -1, 63, 0])
    cache = torch.full((nb, bs, C + R), 7.0, dtype=dtype, device=device)
    cs = ops.rope_cos_sin_table(rot, 512, 300.0).to(device)
    cq, rows = ap.latent_prepare(a, 0, kv0, kr, rot, None, cw.to(device), eps, cs, pos.to(device), slots.to(device), cache, C, 0, True)
    assert cq is None
    close(rows[:, :kr], oracle.rms(ref[:, kv0:kv0 + kr], eps) * cw.double(), TOL[dtype])
    assert not rows[:, kr:C].any() and not rows[:, C + rot:].any()
    ok = slots >= 0
    assert torch.equal(cache.view(-1, C + R)[slots[ok].to(device)], rows[ok.to(device)])
    assert int((cache == 7).all(-1).sum()) == nb * bs - int(ok.sum())
    # the key part turns by halves; its columns are the pairs of neighbours, even ones first
    order = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2)])
    full = torch.zeros(501, 1, rot, dtype=torch.double)
    full[pos[:, None], 0, order] = ref[:, kv0 + kr:kv0 + kr + rot]
    close(rows[:, C:C + rot], oracle.rotate_neighbours(full, rot, 300.0)[pos, 0][:, order], TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,C,R", [(4, 64, 16), (20, 96, 32), (3, 16, 8), (16, 512, 64), (5, 512, 64), (2, 200, 56), (100, 512, 64), (2, 600, 8)])
def test_sink_in_latent_space(device, dtype, H, C, R):
    """Sinks far below, among and far above the scores, short and long sequences (one or several parts of the keys)."""
    if device == "cpu" and H > 5:
        pytest.skip("covered by the other sizes")
    lens, portions = [1, 65, 700, 130, 2], [1, 1, 2, 3, 1]
    q, kc, _, a, cu, ks, _, qs = paged_case(lens, portions, H, 1, C + R, 8, 64, dtype, device, seed=C)
    a["seq_lens"] = (a["positions"] + 1).int()
    scale, sink = 1.5 / math.sqrt(C + R), torch.linspace(-6.0, 12.0, H)
    for longest in (max(lens), 64):         # decides how many parts there are
        got = ap.latent_attention(q.contiguous(), kc.squeeze(2), C, scale=scale, sink=sink.to(device), max_seq_len=longest, **a)
        want = want_attention(lens, portions, ks, [k[..., :C] for k in ks], qs, scale, 0, sink=sink.double()).view(-1, H, C)
        for h in range(H):
            close(got[:, h], want[:, h], TOL[dtype] * 2)


@pytest.mark.gpu
@pytest.mark.parametrize("H,d1,d2,dv", [(4, 128, 64, 128), (3, 40, 16, 88), (2, 8, 8, 8), (5, 64, 64, 72), (2, 104, 40, 128)])
def test_sink_over_projected_keys(H, d1, d2, dv):
    portions, ctx = [130, 20, 300, 9], [0, 200, 69, 1]
    lens = [c + n for c, n in zip(ctx, portions)]
    T, K = sum(portions), sum(lens)
    q, qd = acts(rnd(T, H * (d1 + d2), seed=1), BF16, "cuda")
    kv, kd = acts(rnd(K, H * (d1 + dv), seed=2), BF16, "cuda")
    k2, k2d = acts(rnd(K, d2, seed=3), BF16, "cuda", d2 + 16)
    q0 = torch.tensor([0, *portions]).cumsum(0).tolist()
    k0 = torch.tensor([0, *lens]).cumsum(0).tolist()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")      # noqa: E731
    sink, scale = torch.linspace(-5.0, 9.0, H), 1.6 / math.sqrt(d1 + d2)
    out = ap.latent_prefill(q.view(T, H, d1 + d2), kv, k2[:, :d2], d1=d1, dv=dv, q_start=i32(q0[:-1]), q_end=i32(q0[1:]), k_start=i32(k0[:-1]),
                            k_end=i32(k0[1:]), max_q=300, scale=scale, sink=sink.cuda()).view(T, H, dv)
    for i, (n, m) in enumerate(zip(portions, lens)):
        rows = kd[k0[i]:k0[i + 1]].view(m, H, d1 + dv)
        full = torch.zeros(m, H, d1 + d2, dtype=torch.double)
        full[m - n:] = qd[q0[i]:q0[i + 1]].view(n, H, d1 + d2)
        k = torch.cat([rows[..., :d1], k2d[k0[i]:k0[i + 1], None].expand(m, H, d2)], -1)
        s = torch.einsum("ihd,jhd->hij", full, k) * scale
        want = oracle.softmax_values(s, oracle.causal_mask(m), rows[..., d1:], sink.double())[m - n:]
        for h in range(H):
            close(out[q0[i]:q0[i + 1], h], want[:, h], TOL[BF16] * 2)


def test_rotated_rows_are_stored_even_ones_first():
    m = LatentAttention(LatentSpec(2, 3, 4, 5, 0, 6, 1.0, gate=False, rot_pairs=True), 7, 1e-5, dtype=F32)
    t = m.checkpoint_targets()
    assert set(t) == {"q", "dkv", "dkv.norm", "uk", "uv", "o"}
    t["q"][0](torch.arange(14.0)[:, None].expand(14, 7))
    assert m.in_proj.weight[:m.kv0, 0].view(2, 16)[:, [0, 1, 2, 8, 9, 10, 11]].tolist() == [[0, 1, 2, 3, 5, 4, 6], [7, 8, 9, 10, 12, 11, 13]]
    t["dkv"][0](torch.arange(10.0)[:, None].expand(10, 7))
    assert m.in_proj.weight[m.kv0:m.kv0 + 10, 0].tolist() == [0, 1, 2, 3, 4, 5, 6, 8, 7, 9]


# ----------------------------------------------------------------------------- gated linear attention
GLA_SIZES = [(3, 16, 24, 5.0), (2, 64, 64, 16.0), (1, 40, 136, 0.5), (2, 128, 32, 8.0), (2, 7, 13, 2.0), (1, 256, 72, 16.0), (4, 32, 200, 1.0), (1, 300, 16, 16.0),
             (1, 8, 8, 1.0)]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,N,P,tau", GLA_SIZES)
@pytest.mark.parametrize("cut", range(len(CUTS)))
def test_gated_linear_attention(device, dtype, H, N, P, tau, cut):
    """Decays from almost one to almost zero in neighbouring channels, then norm and gate."""
    if device == "cpu" and (cut in (0, 3) or N > 70):
        pytest.skip("covered by the other sizes")
    lens = [300, 130]
    data = [{k: rnd(lens[r], H * (N if k in "qkz" else P), seed=10 * r + i) for i, k in enumerate(("q", "k", "z", "v", "gate"))} for r in range(2)]
    b = (torch.linspace(-6.0, 9.0, H * N)[torch.randperm(H * N, generator=torch.Generator().manual_seed(5))] * min(tau, 4.0)).contiguous()
    nw, want = 1 + 0.3 * rnd(P, seed=42), []
    for d in data:
        T = d["q"].shape[0]
        s = {k: d[k].to(dtype).double().view(T, H, -1) for k in ("q", "k", "v", "gate")}
        alpha = oracle.gla_decay(d["z"].double() + b.double(), tau).view(T, H, N)
        o, _ = oracle.gla_scan(s["q"] * N ** -0.5, s["k"], s["v"], alpha)
        want.append((oracle.rms(o, 1e-4) * nw.double() * oracle.silu(s["gate"])).reshape(T, H * P))
    S = torch.full((3, H, P, N), 5.0, device=device)
    n, m = ll.pad8(H * N), ll.pad8(H * P)

    def call(rows, kw, span):
        part = lambda k: torch.cat([data[r][k][a:e] for r, a, e in rows])      # noqa: E731
        u = torch.zeros(part("q").shape[0], 2 * n + 2 * m)
        for k, at in (("q", 0), ("k", n), ("v", 2 * n), ("gate", 2 * n + m)):
            u[:, at:at + part(k).shape[1]] = part(k)
        u = u.to(dtype).to(device)
        z = torch.zeros(u.shape[0], n)
        z[:, :H * N] = part("z")
        kw = {k: v.to(device) if v is not None else None for k, v in kw.items()}
        y = ms.gla_scan(u[:, :H * N], u[:, n:n + H * N], u[:, 2 * n:2 * n + H * P], z.to(device), b.to(device), 1 / tau, S, H=H, P=P, N=N, **kw, **span)
        out = torch.empty(u.shape[0], m, dtype=dtype, device=device)
        ms.head_norm(y, u[:, 2 * n + m:], nw.repeat(H).to(device), out, H=H, P=P, eps=1e-4, act="silu")
        return out[:, :H * P]

    for got, w in zip(by_cuts(CUTS[cut], call), want):
        close(got, w[:got.shape[0]], TOL[dtype] * 2)
        d = (got.double() - w[:got.shape[0]]).pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
        assert float(d.max()) < TOL[dtype] * 2
    assert (S[1] == 5).all()


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_pair_in_the_gated_state(device, dtype):
    """One key / value pair hundreds of tokens back, everything since then orthogonal to the query; a slow channel still holds it, its
    own token reads it undecayed."""
    H, N, P, T = 1, 64, 64, 700
    q, k, v = rnd(T, N, seed=1) * 0.3, rnd(T, N, seed=2), rnd(T, P, seed=3)
    k[:, :8] = 0
    k[5] = 0
    k[5, 3] = 8.0
    q[-1] = q[5] = 0
    q[-1, 3] = q[5, 3] = 6.0
    dev = lambda t: t.to(dtype).to(device)      # noqa: E731
    S = torch.ones(1, H, P, N, device=device)
    y = ms.gla_scan(dev(q), dev(k), dev(v), torch.zeros(T, N, device=device), torch.full((N,), 4.0, device=device), 1 / 16, S, H=H, P=P, N=N,
                    positions=torch.arange(T, device=device), state_slots=torch.zeros(1, dtype=torch.int32, device=device),
                    cu_q=torch.tensor([0, T], dtype=torch.int32, device=device), min_q=T, max_q=T)
    alpha = (1 / (1 + math.exp(-4.0))) ** (1 / 16)
    for t, steps in ((5, 0), (T - 1, T - 6)):
        want = v[5].to(dtype).double() * 48 / 8 * alpha ** steps
        assert float((y[t].double().cpu() - want).norm() / want.norm()) < max(2 * TOL[dtype], 2e-4)


# ----------------------------------------------------------------------------- experts
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H,ff,sff,E,top,groups", [(1, 16, 8, 16, 4, 2, (2, 1)), (70, 64, 128, 256, 8, 3, (4, 2)), (9, 37, 13, 21, 5, 5, None),
                                                     (150, 72, 24, 0, 6, 1, (3, 1)), (300, 64, 128, 40, 9, 4, (3, 2)), (40, 24, 16, 8, 12, 4, (2, 1)),
                                                     (33, 24, 8, 8, 4, 2, (4, 3))])
def test_group_limited_mixture(device, dtype, T, H, ff, sff, E, top, groups):
    m = {"router": {"experts": E, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None}, "expert": {"ff": ff},
         "shared": {"ff": sff} if sff else None}
    w = {"p.router": rnd(E, H, seed=1, scale=1.5 / math.sqrt(H)).to(dtype)}
    for i, (e, n) in enumerate([(f"e{e}.", ff) for e in range(E)] + ([("shared.", sff)] if sff else [])):
        for j, (c, o, k) in enumerate((("gate", n, H), ("up", n, H), ("down", H, n))):
            w[f"p.{e}{c}"] = rnd(o, k, seed=10 + 3 * i + j, scale=1.5 / math.sqrt(k)).to(dtype)
    g = groups or (1, 1)
    layer = ExpertMixture(ExpertsSpec(E, top, ff, shared_ff=sff, act="swiglu", weighting="sigmoid", groups=g[0], keep_groups=g[1]), H, dtype=dtype,
                          device=device)
    targets = layer.checkpoint_targets()
    assert {"p." + k for k in targets} == set(w)
    for name, (p, r0, rows, cols) in targets.items():
        (p.data[r0:r0 + rows] if cols is None else p.data[r0:r0 + rows, :cols]).copy_(w["p." + name])
    x, xd = acts(rnd(T, H, seed=4), dtype, device, ll.pad8(H))
    wd = {k: v.double() for k, v in w.items()}
    z = xd @ wd["p.router"].T
    ids, _ = oracle.route(z, m["router"])
    # rows in which a small change of the logits moves the choice are left out
    same = torch.ones(T, dtype=torch.bool)
    for s in range(8):
        other, _ = oracle.route(z + 1e-2 * rnd(T, E, seed=70 + s).double(), m["router"])
        same &= (other.sort(-1).values == ids.sort(-1).values).all(-1)
    assert same.float().mean() > 0.7
    got = layer(x)
    assert torch.equal(got.ids.cpu().long().sort(-1).values[same], ids.sort(-1).values[same])
    close(got.total()[same.to(device), :H], oracle.mixture(xd, wd, "p.", m)[same], TOL[dtype] * 2)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_groups_limit_the_choice(device, dtype):
    """The best expert stands in a group whose two best are worse together than another group's."""
    z = torch.tensor([[4.0, -9.0, -9.0, 1.0, 2.0, 0.5]], device=device)
    ids, w = ops.router_topk(z, 2, mode="sigmoid", n_group=2, topk_group=1, group_mode="top2sum")
    assert ids.tolist() == [[4, 3]]
    assert w[0].tolist() == pytest.approx(torch.sigmoid(torch.tensor([2.0, 1.0])).tolist(), rel=1e-5)
    assert ops.router_topk(z, 2, mode="sigmoid", n_group=2, topk_group=2, group_mode="top2sum")[0].tolist() == [[0, 4]]

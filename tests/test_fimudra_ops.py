"""Every op that the Fimudra design adds, alone, against the plain implementation: CPU references and CUDA kernels, fp32 and
bf16, sizes on and off the tensor-core paths, requests cut into portions, slots that hold another request's leftovers."""
import math

import pytest
import torch

import fimudra_oracle as oracle
from omni_infer_b200 import ops
from omni_infer_b200.layers.common import ClampedGLUMLP
from omni_infer_b200.layers.moe import ExpertMixture
from omni_infer_b200.models.config import ExpertsSpec
from omni_infer_b200.ops import layer_list as ll
from omni_infer_b200.ops import matrix_state as ms
from omni_infer_b200.ops import streams as st
from test_layer_list_ops import BF16, F32, RUNS, TOL, acts, close, paged_case, rnd


@pytest.fixture(autouse=True)
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


# ----------------------------------------------------------------------------- residual streams
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H,S", [(1, 8, 1), (5, 37, 2), (3, 200, 3), (2, 2052, 4), (4, 24, 6)])
def test_streams(device, dtype, T, H, S):
    """Update from the old streams, indexed [from, to], the sum and the layer norm (far from zero mean, eps counts)."""
    ld, eps = ll.pad8(H), 1e-3
    x = torch.zeros(T, S, ld)
    x[:, :, :H] = rnd(T, S, H, seed=1, scale=0.05) + 0.3
    mix, out, inw, w = rnd(S, S, seed=2), rnd(S, seed=3), rnd(S, seed=4), 1 + 0.2 * rnd(H, seed=5)
    y, yd = acts(rnd(T, H, seed=6, scale=0.05), dtype, device, ld)
    want_x = oracle.spread_streams(x[:, :, :H].double(), mix.double(), out.double(), yd)
    want_h = oracle.layer_norm(oracle.gather_streams(want_x, inw.double()), w.double(), eps)
    dev = lambda *ts: [t.to(device) for t in ts]      # noqa: E731
    for last in (False, True):
        xd, m, o, i, wd = dev(x.clone(), mix, out, inw, w)
        h = st.stream_step(xd, y, m, o, i, wd, eps, dtype, last=last)
        close(h[:, :H], want_h, TOL[dtype])
        assert h.dtype == dtype and not h[:, H:].any()
        if not last:
            close(xd[:, :, :H], want_x, 2e-6)
    table, td = acts(rnd(11, H, seed=7), dtype, device, ld)
    ids = torch.tensor([7, 0, 10, 3, 7][:T], device=device)
    xs, h = st.embed_streams(ids, table, H, 3.5, inw.to(device), w.to(device), eps)
    e = td[ids.cpu()] * 3.5
    close(xs[:, :, :H], e[:, None].repeat(1, S, 1), 2e-6)
    close(h[:, :H], oracle.layer_norm(e * float(inw.double().sum()), w.double(), eps), TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
def test_expert_parts_are_summed_into_the_streams(device, dtype):
    T, H, S, k, E, eps = 6, 40, 2, 3, 5, 1e-5
    g = torch.Generator().manual_seed(1)
    ids = torch.stack([torch.randperm(E + 3, generator=g)[:k] for _ in range(T)]).int()
    ids[4] = torch.tensor([5, 7, 6])                   # identity experts only
    ids[5] = -1                                        # padding row
    w = torch.rand(T, k, generator=g)
    y, yd = acts(rnd(T * k, H, seed=2), dtype, device)
    row_of = torch.where((ids >= 0) & (ids < E), torch.randperm(T * k, generator=g).view(T, k).int(), -1)
    h, hd = acts(rnd(T, H, seed=3), dtype, device)
    sh, shd = acts(rnd(T, H, seed=4), dtype, device)
    for shared in (sh, None):
        total = torch.zeros(T, H, dtype=torch.double) if shared is None else shd.clone()
        for t in range(T):
            for j in range(k):
                if row_of[t, j] >= 0:
                    total[t] += yd[row_of[t, j]]
                elif ids[t, j] >= E:
                    total[t] += w[t, j].double() * hd[t]
        x, mix, out, inw, nw = rnd(T, S, H, seed=5), rnd(S, S, seed=6), rnd(S, seed=7), rnd(S, seed=8), torch.ones(H)
        want = oracle.spread_streams(x.double(), mix.double(), out.double(), total)
        xd = x.clone().to(device)
        es = st.ExpertSum(y, row_of.flatten().to(device), ids.to(device), w.to(device), E, h, shared)
        close(es.total(), total, 2e-6)
        st.stream_step(xd, es, mix.to(device), out.to(device), inw.to(device), nw.to(device), eps, dtype)
        close(xd, want, 2e-6)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H", [16, 37, 264])
def test_token_shift_across_cuts(device, dtype, H):
    """Portions of several requests, single tokens, a request in a slot that holds another one's leftovers."""
    mu = torch.rand(5, H, generator=torch.Generator().manual_seed(1))
    seqs = [rnd(9, H, seed=2), rnd(4, H, seed=3), rnd(6, H, seed=4)]
    part, ld = (H + 63) // 64 * 64, ll.pad8(H)
    state = torch.full((3, H), 9.0, dtype=dtype, device=device)
    slots, at, got = [2, 0, 1], [0, 0, 0], [[], [], []]
    want = []
    for s in seqs:
        d = s.to(dtype).double()
        want.append(torch.stack([d + (oracle.token_shift(d) - d) * m.double() for m in mu], 1))
    for step in ([(0, 3), (2, 2)], [(1, 1), (0, 1), (2, 1)], [(0, 5), (1, 3)], [(2, 3)]):
        x, _ = acts(torch.cat([seqs[r][at[r]:at[r] + n] for r, n in step]), dtype, device, ld)
        pos = torch.cat([torch.arange(at[r], at[r] + n) for r, n in step]).to(device)
        ss = torch.tensor([slots[r] for r, _ in step], dtype=torch.int32, device=device)
        single = all(n == 1 for _, n in step)
        cu = torch.tensor([0] + [n for _, n in step]).cumsum(0).int().to(device)
        q2s = torch.tensor([i for i, (_, n) in enumerate(step) for _ in range(n)], dtype=torch.int32, device=device)
        o = st.token_shift(x, mu.to(device), state, part, positions=pos, state_slots=ss, q_to_seq=q2s, cu_q=None if single else cu)
        assert not o[:, :, H:].any()
        a = 0
        for r, n in step:
            got[r].append(o[a:a + n, :, :H].cpu())
            a, at[r] = a + n, at[r] + n
    for r in range(3):
        close(torch.cat(got[r]), want[r], TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
def test_tanh_keeps_sixteen_bits(device, dtype):
    a = rnd(7, 24, seed=1, scale=2.0)
    o = st.tanh_split(a.to(device), 19, dtype)
    want = torch.tanh(a[:, :19].double())
    half = o.shape[1] if dtype == F32 else o.shape[1] // 2
    got = o.double() if dtype == F32 else o[:, :half].double() + o[:, half:].double()
    close(got[:, :19], want, 2e-6 if dtype == F32 else 2e-5)
    assert half == 24 and not o[:, 19:24].any() and not o[:, half + 19:].any()


# ----------------------------------------------------------------------------- attention with a sink
SINK_SHAPES = [(4, 2, 64, 64), (2, 1, 72, 104), (8, 2, 128, 128), (3, 1, 9, 5), (6, 2, 192, 40), (20, 1, 32, 32), (2, 2, 200, 136)]


def sink_want(lens, portions, ks, vs, qs, scale, sink, out_scale):
    out = []
    for n, m, k, v, q in zip(lens, portions, ks, vs, qs):
        full = torch.zeros(n, *q.shape[1:], dtype=torch.double)
        full[n - m:] = q
        out.append(oracle.sink_attention(full, k, v, scale, sink.double())[n - m:].reshape(m, -1) * out_scale)
    return torch.cat(out)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv", SINK_SHAPES)
@pytest.mark.parametrize("decode", [False, True], ids=["portion", "decoded"])
def test_attention_with_a_sink(device, dtype, H, G, d, dv, decode):
    """Sinks from far below to far above the scores; the result scaled and written into wider rows."""
    lens = [5, 200, 64, 321, 1] if not decode else [1, 63, 64, 65, 700]
    portions = [5, 130, 1, 2, 1] if not decode else [1] * 5
    scale, out_scale = 1.7 / math.sqrt(d), 0.7
    sink = torch.linspace(-6.0, 9.0, H)
    q, kc, vc, a, cu, ks, vs, qs = paged_case(lens, portions, H, G, d, dv, 64, dtype, device, seed=d)
    want = sink_want(lens, portions, ks, vs, qs, scale, sink, out_scale)
    for any_shape in (False, True):
        out = torch.full((q.shape[0], ll.pad8(H * dv) + 8), 7.0, dtype=dtype, device=device)
        got = ll.paged_attention(q, kc, vc, scale=scale, cu_q=None if decode else cu, max_q=max(portions), max_seq_len=max(lens),
                                 sink=sink.to(device), out_scale=out_scale, out=out, any_shape=any_shape, **a)
        assert got is out and (out[:, ll.pad8(H * dv):] == 7).all()
        for h in range(H):      # per head: a large sink makes its head's output small
            close(got[:, h * dv:(h + 1) * dv], want[:, h * dv:(h + 1) * dv], TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["portion", "decoded"])
@pytest.mark.parametrize("at", [0, 63, 64, 127, 128, 575])
def test_far_key_beside_a_sink(device, dtype, decode, at):
    """One key, at the start or at a page's border, outweighs hundreds of others; the sink takes a part of its weight."""
    H, G, d, dv, n = 4, 2, 64, 64, 577
    m = 1 if decode else 3
    q, kc, vc, a, cu, ks, vs, qs = paged_case([n], [m], H, G, d, dv, 64, dtype, device, seed=at, spike=[(0, n - 1, at, 2.0)])
    scale = 1 / math.sqrt(d)
    sink = (qs[0][-1].view(G, 2, d) * ks[0][at].view(G, 1, d)).sum(-1).view(-1).float() * scale - 0.5
    got = ll.paged_attention(q, kc, vc, scale=scale, cu_q=None if decode else cu, max_q=m, max_seq_len=n, sink=sink.to(device), **a)
    want = sink_want([n], [m], ks, vs, qs, scale, sink, 1.0)
    close(got[-1:], want[-1:], TOL[dtype])
    without = sink_want([n], [m], ks, vs, qs, scale, torch.full((H,), -80.0), 1.0)
    assert float((want[-1] - without[-1]).abs().max() / want[-1].abs().max()) > 0.2, "the case does not show the sink"


def test_llama3_frequencies():
    """Long wavelengths slowed, short ones kept, the band between blended: every branch is taken."""
    for dims, base, s in ((64, 1e4, dict(factor=4.0, low=1.0, high=4.0, original=512)), (20, 500.0, dict(factor=8.0, low=0.5, high=2.0, original=64))):
        t = ops.rope_cos_sin_table(dims, 3000, base, {"type": "llama3", "factor": s["factor"], "low_freq_factor": s["low"],
                                                      "high_freq_factor": s["high"], "original_max_position_embeddings": s["original"]})
        f = torch.tensor([oracle.frequency(i, dims, base, s) for i in range(dims // 2)], dtype=torch.double)
        raw = torch.tensor([oracle.frequency(i, dims, base, None) for i in range(dims // 2)], dtype=torch.double)
        assert (f == raw).any() and (f == raw / s["factor"]).any() and ((f < raw) & (f > raw / s["factor"])).any()
        a = torch.arange(3000, dtype=torch.double)[:, None] * f
        assert (t.double() - torch.cat([a.cos(), a.sin()], 1)).abs().max() < 1e-6


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv,rot", [(4, 2, 16, 24, 8), (3, 1, 9, 5, 6), (2, 2, 64, 64, 64)])
def test_rotation_and_cache_write_without_norms(device, dtype, H, G, d, dv, rot):
    T, bs, nb = 5, 16, 5
    n = (H + G) * d + G * dv
    qkv, ref = acts(rnd(T, n, seed=1), dtype, device, ll.pad8(n) + 8)
    pos, slots = torch.tensor([0, 1, 300, 17, 900]), torch.tensor([3, 70, 11, -1, 0])
    sc = dict(factor=4.0, low=1.0, high=4.0, original=256)
    cs = ops.rope_cos_sin_table(rot, 1024, 1e3, {"type": "llama3", "factor": 4.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                                                 "original_max_position_embeddings": 256}).to(device)
    kc, vc = torch.zeros(nb, bs, G, d, dtype=dtype, device=device), torch.zeros(nb, bs, G, dv, dtype=dtype, device=device)
    ll.qk_norm_rope_cache(qkv, H, G, d, dv, None, None, 0.0, cs, rot, pos.to(device), slots.to(device), kc, vc)
    r = dict(dims=rot, base=1e3, scaling=sc)
    close(qkv[:, : H * d].reshape(T, H, d), oracle.rotate(ref[:, : H * d].view(T, H, d), pos, r), TOL[dtype])
    ok = slots >= 0
    close(kc.view(-1, G, d)[slots[ok].to(device)], oracle.rotate(ref[:, H * d:(H + G) * d].view(T, G, d), pos, r)[ok], TOL[dtype])
    assert torch.equal(vc.view(-1, G, dv)[slots[ok].to(device)].double().cpu(), ref[ok, (H + G) * d: n].view(-1, G, dv))


# ----------------------------------------------------------------------------- matrix memory and WKV, by cuts
CUTS = [[[(0, 300)], [(1, 130)]], [[(0, 1), (1, 2)], [(0, 129), (1, 1)], [(0, 2), (1, 127)], [(0, 168)]],
        [[(0, 128), (1, 64)], [(0, 1), (1, 1)], [(0, 7), (1, 9)], [(0, 161), (1, 1)], [(0, 3), (1, 55)]],
        [[(0, 1)]] * 3 + [[(1, 1), (0, 1)]] * 130 + [[(0, 167)]]]


def by_cuts(cuts, call):
    """``call(rows [(request, first, end)], kwargs)`` for every step; requests 0 and 1 live in slots 2 and 0, row 3 of a step of
    single tokens is padding."""
    at, got = [0, 0], [[], []]
    for step in cuts:
        rows = [(r, at[r], at[r] + n) for r, n in step]
        single = all(n == 1 for _, n in step)
        slots, lens, pos = [[2, 0][r] for r, _ in step], [n for _, n in step], [torch.arange(a, b) for _, a, b in rows]
        if single and len(step) == 2:
            slots, lens, pos, rows = slots + [-1], lens + [1], pos + [torch.zeros(1, dtype=torch.long)], rows + [(0, 0, 1)]
        kw = dict(positions=torch.cat(pos), state_slots=torch.tensor(slots, dtype=torch.int32),
                  cu_q=None if single else torch.tensor([0] + lens).cumsum(0).int())
        o = call(rows, kw, dict(min_q=min(lens), max_q=max(lens)))
        a = 0
        for (r, n) in step:
            got[r].append(o[a:a + n].cpu())
            a, at[r] = a + n, at[r] + n
    return [torch.cat(g) for g in got]


MEM_SIZES = [(2, 8, 8), (3, 40, 56), (2, 64, 128), (1, 128, 72), (2, 13, 9), (1, 160, 40), (2, 72, 64)]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,N,P", MEM_SIZES)
@pytest.mark.parametrize("cut", range(len(CUTS)))
def test_matrix_memory(device, dtype, H, N, P, cut):
    if device == "cpu" and (cut in (0, 3) or N > 70):
        pytest.skip("covered by the other sizes")
    cap, eps = 9.0, 1e-4
    lens = [300, 130]
    f_col = ll.pad8(H)
    data = []
    for r in range(2):
        g = lambda *s, k=0, scale=1.0: rnd(lens[r], *s, seed=10 * r + k, scale=scale)      # noqa: E731
        z = torch.zeros(lens[r], 2 * f_col)
        z[:, :H], z[:, f_col:f_col + H] = g(H, k=1, scale=6.0), g(H, k=2, scale=4.0) + 4
        data.append(dict(q=g(H * N, k=3), k=g(H * N, k=4, scale=0.5), v=g(H * P, k=5), gate=g(H * P, k=6), z=z))
    ib, fb, nw = rnd(H, seed=31) - 1, rnd(H, seed=32) + 1, 1 + 0.3 * rnd(H * P, seed=33)
    want = []
    for d in data:
        T = d["q"].shape[0]
        st_ = {k: d[k].to(dtype).double() for k in ("q", "k", "v", "gate")}
        z = d["z"].double()
        o = oracle.matrix_memory(st_["q"].view(T, H, N) / math.sqrt(N), st_["k"].view(T, H, N), st_["v"].view(T, H, P),
                                 oracle.capped(z[:, :H] + ib.double(), cap),
                                 oracle.log_sigmoid(oracle.capped(z[:, f_col:f_col + H] + fb.double(), cap)))
        want.append(oracle.unit_rms(o, eps).reshape(T, -1) * nw.double() * oracle.sigmoid(st_["gate"]) * 0.6)
    S = torch.full((3, H, P + 1, N), 5.0, device=device)
    m = torch.full((3, H), 4.0, device=device)
    pitch = ll.pad8(H * N)

    def call(rows, kw, span):
        part = lambda k: torch.cat([data[r][k][a:b] for r, a, b in rows])      # noqa: E731
        u = torch.zeros(part("q").shape[0], 2 * pitch + 2 * ll.pad8(H * P))
        offs = (0, pitch, 2 * pitch, 2 * pitch + ll.pad8(H * P))
        for k, o in zip(("q", "k", "v", "gate"), offs):
            u[:, o:o + part(k).shape[1]] = part(k)
        u = u.to(dtype).to(device)
        kw = {k: v.to(device) if v is not None else None for k, v in kw.items()}
        gates = ms.mlstm_gates(part("z").to(device), f_col, ib.to(device), fb.to(device), cap, m,
                               chunks=device == "cuda" and ms.mlstm_chunked(dtype, N, P), **kw)
        y = ms.mlstm_scan(u[:, :H * N], u[:, offs[1]:offs[1] + H * N], u[:, offs[2]:offs[2] + H * P], gates, S, H=H, P=P, N=N, **kw, **span)
        out = torch.empty(u.shape[0], ll.pad8(H * P), dtype=dtype, device=device)
        ms.head_norm(y, u[:, offs[3]:], nw.to(device), out, H=H, P=P, eps=eps, act="sigmoid", scale=0.6, gates=gates)
        return out[:, :H * P]

    for got, w in zip(by_cuts(CUTS[cut], call), want):
        close(got, w[:got.shape[0]], TOL[dtype] * 2)
        # per row: one wrong token must not hide behind the largest row (rounding of y before its norm stays relative to the row)
        d = (got.double() - w[:got.shape[0]]).pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
        assert float(d.max()) < TOL[dtype] * 2
    assert (S[1] == 5).all() and (m[1] == 4).all()


WKV_SIZES = [(2, 8), (3, 32), (2, 64), (1, 128), (2, 13), (1, 160), (2, 72), (1, 48)]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,N", WKV_SIZES)
@pytest.mark.parametrize("cut", range(len(CUTS)))
def test_wkv(device, dtype, H, N, cut):
    """Decays from almost one to almost zero in neighbouring channels."""
    if device == "cpu" and (cut in (0, 3) or N > 70):
        pytest.skip("covered by the other sizes")
    lens = [300, 130]
    n = H * N
    data = [{k: rnd(lens[r], n, seed=10 * r + i) for i, k in enumerate(("r", "k", "v", "z", "gate"))} for r in range(2)]
    w0 = torch.linspace(-9.0, 3.0, n)[torch.randperm(n, generator=torch.Generator().manual_seed(5))].contiguous()
    u, nw = rnd(n, seed=41), 1 + 0.3 * rnd(n, seed=42)
    want = []
    for d in data:
        T = d["r"].shape[0]
        s = {k: d[k].to(dtype).double().view(T, H, N) for k in ("r", "k", "v", "gate")}
        dec = torch.exp(-torch.exp(d["z"].double() + w0.double())).view(T, H, N)
        o, _ = oracle.wkv_scan(s["r"], s["k"], s["v"], dec, u.double().view(H, N))
        want.append((oracle.unit_rms(o, 1e-4) * (s["gate"] * oracle.sigmoid(s["gate"]))).reshape(T, n) * nw.double())
    S = torch.full((3, H, N, N), 5.0, device=device)
    block = ll.pad8(n)

    def call(rows, kw, span):
        part = lambda k: torch.cat([data[r][k][a:b] for r, a, b in rows])      # noqa: E731
        p = torch.zeros(part("r").shape[0], 4, block)
        for i, k in enumerate(("r", "k", "v", "gate")):
            p[:, i, :n] = part(k)
        p = p.to(dtype).to(device)
        z = torch.zeros(p.shape[0], block)
        z[:, :n] = part("z")
        kw = {k: v.to(device) if v is not None else None for k, v in kw.items()}
        y = ms.wkv_scan(p[:, 0, :n], p[:, 1, :n], p[:, 2, :n], z.to(device), w0.to(device), u.to(device), S, H=H, N=N, **kw, **span)
        out = torch.empty(p.shape[0], block, dtype=dtype, device=device)
        ms.head_norm(y, p[:, 3], nw.to(device), out, H=H, P=N, eps=1e-4, act="silu")
        return out[:, :n]

    for got, w in zip(by_cuts(CUTS[cut], call), want):
        close(got, w[:got.shape[0]], TOL[dtype] * 2)
        d = (got.double() - w[:got.shape[0]]).pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
        assert float(d.max()) < TOL[dtype] * 2
    assert (S[1] == 5).all()


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_pair_in_the_matrix_states(device, dtype):
    """One key / value pair hundreds of tokens back, everything since then orthogonal to the query: it is all that is read."""
    H, N, P, T = 1, 64, 64, 700
    q, k, v = rnd(T, N, seed=1) * 0.3, rnd(T, N, seed=2), rnd(T, P, seed=3)
    k[:, :8] = 0
    k[5] = 0
    k[5, 3] = 8.0
    q[-1] = 0
    q[-1, 3] = 6.0
    dev = lambda t: t.to(dtype).to(device)      # noqa: E731
    kw = dict(positions=torch.arange(T, device=device), state_slots=torch.zeros(1, dtype=torch.int32, device=device),
              cu_q=torch.tensor([0, T], dtype=torch.int32, device=device))
    z = torch.full((T, 16), -1.0)
    z[:, 8] = 8.0
    zero = torch.zeros(1, device=device)
    S, m = torch.ones(1, H, P + 1, N, device=device), torch.ones(1, H, device=device)
    gates = ms.mlstm_gates(z.to(device), 8, zero, zero, 20.0, m, chunks=device == "cuda", **kw)
    y = ms.mlstm_scan(dev(q), dev(k), dev(v), gates, S, H=H, P=P, N=N, **kw, min_q=T, max_q=T)
    o = y[-1].double().cpu() / max(abs(float(gates.den[-1, 0])), math.exp(-float(gates.m[-1, 0])))
    assert float((o - v[5].to(dtype).double()).norm() / v[5].norm()) < 5 * TOL[dtype]
    S = torch.ones(1, H, P, N, device=device)
    y = ms.wkv_scan(dev(q), dev(k), dev(v), torch.zeros(T, N, device=device), torch.full((N,), -11.0, device=device),
                    torch.zeros(N, device=device), S, H=H, N=N, **kw, min_q=T, max_q=T)
    want = v[5].to(dtype).double() * 48 * math.exp(-math.exp(-11.0)) ** (T - 7)
    # hundreds of fp32 products with a decay next to one
    assert float((y[-1].double().cpu() - want).norm() / want.norm()) < max(2 * TOL[dtype], 2e-4)


# ----------------------------------------------------------------------------- experts
def mixture_weights(m, H, seed=0):
    n = m["router"]["experts"] + m["router"]["identity"]
    w = {"p.router": rnd(n, H, seed=seed, scale=1.5 / math.sqrt(H)), "p.correction": rnd(n, seed=seed + 1, scale=0.3)}
    mats = [(f"e{e}", m["expert"]["ff"]) for e in range(m["router"]["experts"])] + ([("shared", m["shared"]["ff"])] if m.get("shared") else [])
    for i, (e, ff) in enumerate(mats):
        w[f"p.{e}.gate"], w[f"p.{e}.up"] = rnd(ff, H, seed=seed + 10 + i, scale=2 / math.sqrt(H)), rnd(ff, H, seed=seed + 60 + i, scale=2 / math.sqrt(H))
        w[f"p.{e}.down"] = rnd(H, ff, seed=seed + 110 + i, scale=1 / math.sqrt(ff))
    return w


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H,ff,sff,E,ident,top", [(1, 16, 8, 16, 3, 1, 2), (70, 64, 128, 256, 8, 4, 3), (9, 37, 13, 21, 5, 0, 5),
                                                    (150, 72, 24, 0, 6, 5, 1), (300, 64, 128, 40, 4, 2, 4)])
def test_expert_mixture(device, dtype, T, H, ff, sff, E, ident, top):
    m = {"router": {"experts": E, "identity": ident, "scale": 1.8, "top": top}, "expert": {"ff": ff, "limit": 1.2},
         "shared": {"ff": sff, "limit": 0.6} if sff else None}
    w = {k: (v if "correction" in k else v.to(dtype)) for k, v in mixture_weights(m, H).items()}
    layer = ExpertMixture(ExpertsSpec(E, top, ff, 1.2, ident, 1.8, sff, 0.6), H, dtype=dtype, device=device)
    for name, (p, r0, rows, cols) in layer.checkpoint_targets().items():
        (p.data[r0:r0 + rows] if cols is None else p.data[r0:r0 + rows, :cols]).copy_(w["p." + name])
    x, xd = acts(rnd(T, H, seed=4), dtype, device, ll.pad8(H))
    wd = {k: v.double() for k, v in w.items()}
    # rows whose last choice and first non-choice lie close together are left out: rounding may swap them
    s = torch.softmax(xd @ wd["p.router"].T, -1) + wd["p.correction"]
    order = s.sort(-1, descending=True).values
    clear = torch.ones(T, dtype=torch.bool) if top == s.shape[1] else (order[:, top - 1] - order[:, top]) > 2e-3
    assert clear.float().mean() > 0.8
    want = oracle.expert_mixture(xd, wd, "p.", m)
    got = layer(x)
    close(got.total()[clear.to(device), :H], want[clear], TOL[dtype] * 2)
    assert int((got.ids >= E).sum()) > 0 or not ident or T == 1
    # padding rows take no expert
    if T > 8:
        nv = torch.tensor([T - 3], dtype=torch.int32, device=device)
        ids, _ = ops.router_topk(torch.zeros(T, E + ident, device=device), top, num_valid=nv)
        assert device == "cpu" or (ids[T - 3:] == -1).all()


def test_correction_moves_the_choice_but_not_the_weights():
    z = torch.tensor([[2.0, 1.0, 0.0, -1.0]])
    bias = torch.tensor([-1.0, 0.0, 0.0, 1.0])
    ids, w = ops.router_topk(z, 2, mode="softmax", bias=bias, scale=3.0)
    assert set(ids[0].tolist()) == {3, 1}
    assert torch.allclose(w[0], torch.softmax(z, -1)[0][ids[0].long()] * 3.0)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,K,I", [(1, 16, 8), (70, 64, 128), (9, 40, 13), (130, 72, 256), (33, 24, 136)])
def test_clamped_feed_forward(device, dtype, T, K, I):
    """Gates and ups on both sides of the bounds; only the gate's upper side is bounded."""
    limit = 1.5
    w = {k: v.to(dtype) for k, v in {"m.gate": rnd(I, K, seed=1, scale=3 / math.sqrt(K)), "m.up": rnd(I, K, seed=2, scale=3 / math.sqrt(K)),
                                     "m.down": rnd(K, I, seed=3, scale=1 / math.sqrt(I))}.items()}
    m = ClampedGLUMLP(K, I, limit, dtype=dtype, device=device)
    for name, (p, r0, rows, cols) in m.checkpoint_targets().items():
        p.data[r0:r0 + rows, :cols].copy_(w["m." + name])
    x, xd = acts(rnd(T, K, seed=4), dtype, device, ll.pad8(K))
    wd = {k: v.double() for k, v in w.items()}
    g, u = xd @ wd["m.gate"].T, xd @ wd["m.up"].T
    assert (g > limit).any() and (g < -limit).any() and (u > limit).any() and (u < -limit).any()
    close(m(x)[:, :K], oracle.clamped_glu(xd, wd, "m.", limit), TOL[dtype] * 2)


@pytest.mark.gpu
def test_grouped_products_fp32():
    x, w = rnd(100, 24, seed=1), rnd(3, 20, 24, seed=2)
    start, length = torch.tensor([0, 48, 96], dtype=torch.int32), torch.tensor([40, 0, 3], dtype=torch.int32)
    scale = torch.rand(100, generator=torch.Generator().manual_seed(3))
    got = ops.gemm(x.cuda(), w.cuda(), seg_start=start.cuda(), seg_len=length.cuda(), row_scale=scale.cuda())
    for g in range(3):
        a, n = int(start[g]), int(length[g])
        if n:
            close(got[a:a + n], (x[a:a + n].double() @ w[g].double().T) * scale[a:a + n, None].double(), 2e-6)
    x3, w3 = rnd(9, 3, 16, seed=4), rnd(2, 7, 16, seed=5)
    close(ops.bmm_heads(x3.cuda()[:, :2], w3.cuda()), torch.einsum("thk,hnk->thn", x3[:, :2].double(), w3.double()), 2e-6)

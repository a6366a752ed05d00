"""Every op of the layer-list models against the plain implementation, alone: CPU reference and CUDA kernels, fp32 and
bf16, head and state sizes on and off the tensor-core paths, paged caches with scattered pages, requests cut into portions,
slots that hold another request's leftovers."""
import math

import pytest
import torch

import layer_list_oracle as oracle
from omni_infer_b200 import ops
from omni_infer_b200.ops import layer_list as ll

F32, BF16 = torch.float32, torch.bfloat16
RUNS = [pytest.param("cpu", F32, id="cpu-fp32"),
        pytest.param("cuda", F32, id="cuda-fp32", marks=pytest.mark.gpu),
        pytest.param("cuda", BF16, id="cuda-bf16", marks=pytest.mark.gpu)]
TOL = {F32: 2e-5, BF16: 8e-3}


@pytest.fixture(autouse=True)
def _one_thread():
    """The tensors are tiny: threads only get in each other's way."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def acts(t, dtype, device, ld=None):
    """Activations of ``dtype`` in rows of pitch ``ld`` whose padding is zero; and the values as stored, in double."""
    t = t.to(dtype)
    out = torch.zeros(t.shape[0], ld or t.shape[1], dtype=dtype, device=device)
    out[:, : t.shape[1]] = t.to(device)
    return out, t.double()


def close(got, want, tol, name=""):
    got = got.double().cpu()
    assert torch.isfinite(got).all(), name
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-6))
    assert err < tol, (name, err)


# ----------------------------------------------------------------------------- residual stream, feed-forward, products
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,H", [(1, 8), (5, 37), (3, 200), (2, 4104)])
def test_residual_and_norms(device, dtype, T, H):
    ld = ll.pad8(H)
    x0, w, eps = rnd(T, H, seed=1), 1 + 0.2 * rnd(H, seed=2), 1e-3
    y, yd = acts(rnd(T, H, seed=3, scale=0.05), dtype, device, ld)      # small outputs: eps counts
    x = torch.zeros(T, ld, device=device)
    x[:, :H] = x0.to(device)
    xa = ll.post_norm_add(y, w.to(device), x, eps)
    want = x0.double() + oracle.rms_norm(yd, w.double(), eps)
    close(x[:, :H], want, 2e-6)
    close(xa[:, :H], want, TOL[dtype])
    assert xa.dtype == dtype and not xa[:, H:].any()
    f = ll.rmsnorm_residual(x, w.to(device), eps, dtype)
    close(f[:, :H], oracle.rms_norm(x[:, :H].double().cpu(), w.double(), eps), TOL[dtype])
    assert not f[:, H:].any()
    table, td = acts(rnd(11, H, seed=4), dtype, device, ld)
    ids = torch.tensor([7, 0, 10, 3, 7][:T], device=device)
    x, xa = ll.embed_residual(ids, table)
    assert torch.equal(x[:, :H].double().cpu(), td[ids.cpu()]) and torch.equal(xa[:, :H].double().cpu(), td[ids.cpu()])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,K,I", [(1, 16, 8), (70, 64, 128), (9, 40, 13), (130, 72, 256), (33, 24, 136)])
def test_gated_feed_forward(device, dtype, T, K, I):
    from omni_infer_b200.layers.common import GeGLUMLP
    w = {"m.gate": rnd(I, K, seed=1, scale=2 / math.sqrt(K)), "m.up": rnd(I, K, seed=2, scale=1 / math.sqrt(K)),
         "m.down": rnd(K, I, seed=3, scale=1 / math.sqrt(I))}
    w = {k: v.to(dtype) for k, v in w.items()}
    m = GeGLUMLP(K, I, dtype=dtype, device=device)
    m.gate_up_proj.weight.data[:I, :K] = w["m.gate"].to(device)
    m.gate_up_proj.weight.data[m.block:m.block + I, :K] = w["m.up"].to(device)
    m.down_proj.weight.data[:K, :I] = w["m.down"].to(device)
    m.zero_padding()
    m.down_proj.zero_padding()
    x, xd = acts(rnd(T, K, seed=4), dtype, device, ll.pad8(K))
    close(m(x)[:, :K], oracle.feed_forward(xd, {k: v.double() for k, v in w.items()}, "m."), TOL[dtype] * 2)


@pytest.mark.gpu
@pytest.mark.parametrize("T,N,K", [(1, 1, 1), (3, 70, 17), (65, 130, 200), (128, 64, 1024)])
def test_gemm_fp32(T, N, K):
    x, w = rnd(T, K, seed=1), rnd(N, K, seed=2)
    close(ops.gemm(x.cuda(), w.cuda()), x.double() @ w.double().T, 2e-6)


# ----------------------------------------------------------------------------- q/k norm, rotation, cache
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv,rot,base,factor", [(4, 2, 16, 24, 16, 1e4, 1.0), (3, 1, 9, 5, 6, 500.0, 3.0),
                                                      (2, 2, 8, 8, 0, 1e4, 1.0), (6, 3, 40, 32, 8, 1e6, 8.0), (5, 0, 136, 8, 64, 1e4, 2.0)])
def test_qk_norm_rotation_and_cache_write(device, dtype, H, G, d, dv, rot, base, factor):
    T, eps, bs, nb = 7, 1e-4, 16, 5
    nq, nk, nv = H * d, G * d, G * dv
    qkv, ref = acts(rnd(T, nq + nk + nv, seed=1), dtype, device, ll.pad8(nq + nk + nv))
    qw, kw = 1 + 0.3 * rnd(nq, seed=2), 1 + 0.3 * rnd(max(nk, 1), seed=3)
    pos = torch.tensor([0, 1, 2, 300, 301, 17, 900])
    slots = torch.tensor([3, 70, 11, -1, 0, 79, 33])
    cs = ops.rope_cos_sin_table(rot, 1024, base, {"type": "linear", "factor": factor}).to(device) if rot else None
    kc = torch.full((nb, bs, max(G, 1), d), 7.0, dtype=dtype, device=device)
    vc = torch.full((nb, bs, max(G, 1), dv), 7.0, dtype=dtype, device=device)
    ll.qk_norm_rope_cache(qkv, H, G, d, dv, qw.to(device), kw.to(device), eps, cs, rot, pos.to(device), slots.to(device), kc, vc)
    q = oracle.rms_norm(ref[:, :nq], qw.double(), eps).view(T, H, d)
    q = oracle.rotate(q, pos, rot, base, factor) if rot else q
    close(qkv[:, :nq].reshape(T, H, d), q, TOL[dtype])
    if G:
        k = oracle.rms_norm(ref[:, nq:nq + nk], kw.double(), eps).view(T, G, d)
        k = oracle.rotate(k, pos, rot, base, factor) if rot else k
        ok = slots >= 0
        close(kc.view(-1, G, d)[slots[ok].to(device)], k[ok], TOL[dtype])
        assert torch.equal(vc.view(-1, G, dv)[slots[ok].to(device)].double().cpu(), ref[ok, nq + nk:].view(-1, G, dv))
        untouched = torch.ones(nb * bs, dtype=torch.bool)
        untouched[slots[ok]] = False
        assert (kc.view(-1, G, d)[untouched.to(device)] == 7).all() and (vc.view(-1, G, dv)[untouched.to(device)] == 7).all()


# ----------------------------------------------------------------------------- attention over pages
def paged_case(lens, portions, H, G, d, dv, bs, dtype, device, seed=0, spike=None):
    """Whole sequences of ``lens`` tokens, of which the last ``portions`` are this step's queries; pages scattered."""
    g = torch.Generator().manual_seed(seed)
    nb = [-(-n // bs) for n in lens]
    perm = (torch.randperm(sum(nb) + 3, generator=g) + 1).tolist()
    bt = torch.zeros(len(lens), max(nb) + 2, dtype=torch.int32)
    kc = torch.randn(sum(nb) + 4, bs, G, d, generator=g).to(dtype)
    vc = torch.randn(sum(nb) + 4, bs, G, dv, generator=g).to(dtype)
    qs, ks, vs, pos, seq, slots = [], [], [], [], [], []
    for r, n in enumerate(lens):
        mine = [perm.pop() for _ in range(nb[r])]
        bt[r, : nb[r]] = torch.tensor(mine)
        q = torch.randn(n, H, d, generator=g)
        k = torch.randn(n, G, d, generator=g)
        for (rr, i, j, amount) in spike or ():
            if rr == r:                          # the score of query i with key j stands out, in every head
                k[j] = k[j] * 0.2 + amount * q[i].view(G, H // G, d).mean(1)
        q, k, v = q.to(dtype), k.to(dtype), torch.randn(n, G, dv, generator=g).to(dtype)
        rows = torch.tensor([mine[p // bs] * bs + p % bs for p in range(n)])
        kc.view(-1, G, d)[rows], vc.view(-1, G, dv)[rows] = k, v
        qs.append(q[n - portions[r]:]), ks.append(k.double()), vs.append(v.double())
        pos += list(range(n - portions[r], n))
        seq += [r] * portions[r]
        slots += rows[n - portions[r]:].tolist()
    cu = torch.tensor([0] + list(portions)).cumsum(0)
    T, ld = len(pos), ll.pad8(H * d) + 16
    flat = torch.zeros(T, ld, dtype=dtype)
    flat[:, : H * d] = torch.cat(qs).reshape(T, -1)
    flat = flat.to(device)
    args = dict(positions=torch.tensor(pos), q_to_seq=torch.tensor(seq, dtype=torch.int32), slots=torch.tensor(slots),
                block_table=bt, seq_lens=torch.tensor(lens, dtype=torch.int32))
    args = {k: v.to(device) for k, v in args.items()}
    q3 = flat[:, : H * d].unflatten(1, (H, d))
    return q3, kc.to(device), vc.to(device), args, cu.int().to(device), ks, vs, [q.double() for q in qs]


def paged_want(lens, portions, ks, vs, qs, scale, window):
    out = []
    for n, m, k, v, q in zip(lens, portions, ks, vs, qs):
        full = torch.zeros(n, *q.shape[1:], dtype=torch.double)
        full[n - m:] = q
        out.append(oracle.softmax_attention(full, k, v, scale, window or None)[n - m:].reshape(m, -1))
    return torch.cat(out)


SHAPES = [(4, 2, 64, 64), (2, 1, 72, 104), (8, 2, 128, 128), (4, 4, 16, 24), (3, 1, 9, 5), (6, 2, 192, 40), (20, 1, 32, 32),
          (2, 2, 200, 136)]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv", SHAPES)
@pytest.mark.parametrize("window", [0, 1, 37, 64, 65, 200])
def test_attention_of_portions(device, dtype, H, G, d, dv, window):
    if device == "cpu" and (window in (1, 64, 200) or H * d > 300):
        pytest.skip("covered by the other sizes")
    lens, portions = [5, 200, 64, 321, 130], [5, 130, 1, 2, 129]
    scale = 1.7 / math.sqrt(d)
    q, kc, vc, a, cu, ks, vs, qs = paged_case(lens, portions, H, G, d, dv, 64, dtype, device, seed=d + window)
    got = ll.paged_attention(q, kc, vc, scale=scale, window=window, cu_q=cu, max_q=max(portions), max_seq_len=max(lens), **a)
    close(got[:, : H * dv], paged_want(lens, portions, ks, vs, qs, scale, window), TOL[dtype])
    assert not got[:, H * dv:].any()
    if device == "cuda":
        got = ll.paged_attention(q, kc, vc, scale=scale, window=window, cu_q=cu, max_q=max(portions), any_shape=True, **a)
        close(got[:, : H * dv], paged_want(lens, portions, ks, vs, qs, scale, window), TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,d,dv", SHAPES)
@pytest.mark.parametrize("window,bs", [(0, 64), (1, 16), (40, 64), (64, 128), (300, 16)])
def test_attention_of_single_tokens(device, dtype, H, G, d, dv, window, bs):
    lens = [1, 63, 64, 65, 700, 33]
    scale = 1.7 / math.sqrt(d)
    q, kc, vc, a, _, ks, vs, qs = paged_case(lens, [1] * len(lens), H, G, d, dv, bs, dtype, device, seed=dv + window)
    a["slots"][1], a["seq_lens"][1] = -1, 0                       # a padding row
    want = paged_want(lens, [1] * len(lens), ks, vs, qs, scale, window)
    want[1] = 0
    got = ll.paged_attention(q, kc, vc, scale=scale, window=window, max_seq_len=max(lens), **a)
    close(got[:, : H * dv], want, TOL[dtype])


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["portion", "decoded"])
@pytest.mark.parametrize("window", [48, 64, 100])
def test_window_edge_is_exact(device, dtype, decode, window):
    """A key that dominates every score sits just inside and just outside the last query's window."""
    H, G, d, dv, n = 2, 1, 64, 64, 260
    for dist, inside in ((window - 1, True), (window, False)):
        i = n - 1
        m = 1 if decode else 3
        q, kc, vc, a, cu, ks, vs, qs = paged_case([n], [m], H, G, d, dv, 64, dtype, device, spike=[(0, i, i - dist, 3.0)])
        scale = 1 / math.sqrt(d)
        kw = dict(cu_q=None if decode else cu, max_q=m, max_seq_len=n)
        got = ll.paged_attention(q, kc, vc, scale=scale, window=window, **kw, **a)
        close(got, paged_want([n], [m], ks, vs, qs, scale, window), TOL[dtype])
        v = vs[0][i - dist, 0].repeat(H)
        near = float((got[-1].double().cpu() - v).norm() / v.norm())
        assert (near < 0.2) == inside, near


@pytest.mark.parametrize("device,dtype", RUNS)
def test_very_low_scores_before_the_window_do_not_matter(device, dtype):
    """All scores far below zero, the first key tile of the later queries entirely outside their windows."""
    H, G, d, dv, n, m = 2, 1, 64, 64, 300, 128
    q, kc, vc, a, cu, ks, vs, qs = paged_case([n], [m], H, G, d, dv, 64, dtype, device, seed=5)
    big = 40.0
    q[..., 0], qs[0][..., 0] = big, big
    kc[..., 0], ks[0][..., 0] = -big, -big
    got = ll.paged_attention(q, kc, vc, scale=0.3, window=70, cu_q=cu, max_q=m, max_seq_len=n, **a)
    close(got, paged_want([n], [m], ks, vs, qs, 0.3, 70), max(TOL[dtype], 1e-4))      # scores near -500: fp32 spacing 3e-5


# ----------------------------------------------------------------------------- convolution
def cut(n, sizes):
    """[(start, length)] of a sequence of n tokens cut into portions of the given sizes, repeated."""
    out, a, i = [], 0, 0
    while a < n:
        m = min(sizes[i % len(sizes)], n - a)
        out.append((a, m))
        a, i = a + m, i + 1
    return out


def run_portions(lens, sizes, call):
    """Feeds sequences of ``lens`` tokens in steps; ``call(step)`` gets [(request, start, length)].  Requests join one step
    after another so that every step mixes portions of several lengths and places."""
    plans = [cut(n, sizes[r % len(sizes):] + sizes[: r % len(sizes)]) for r, n in enumerate(lens)]
    step = 0
    while any(plans):
        batch = []
        for r, p in enumerate(plans):
            if p and step >= r:
                a, m = p.pop(0)
                batch.append((r, a, m))
        if batch:
            call(batch)
        step += 1


def batch_md(batch, slots, device):
    cu = torch.tensor([0] + [m for _, _, m in batch]).cumsum(0).int().to(device)
    pos = torch.cat([torch.arange(a, a + m) for _, a, m in batch]).to(device)
    seq = torch.cat([torch.full((m,), i) for i, (_, _, m) in enumerate(batch)]).int().to(device)
    return dict(cu_q=cu, positions=pos, q_to_seq=seq, state_slots=torch.tensor([slots[r] for r, _, _ in batch], dtype=torch.int32).to(device))


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("C,taps", [(16, 4), (40, 3), (13, 2), (24, 1), (9, 7), (520, 4)])
@pytest.mark.parametrize("sizes", [[400], [2, 1, 3], [17, 64, 2, 1, 1]])
def test_convolution_in_portions(device, dtype, C, taps, sizes):
    lens = [40, 1, 23, 9]
    w, b = rnd(C, taps, seed=1), rnd(C, seed=2)
    wt, bd = w.t().contiguous().to(device), b.to(device)
    xs = [acts(rnd(n, C, seed=10 + r), dtype, device, ll.pad8(C) + 8) for r, n in enumerate(lens)]
    state = torch.full((6, taps - 1, C), 9.0, dtype=dtype, device=device)        # leftovers
    slots, got = [4, 0, 3, 1], [[] for _ in lens]

    def call(batch):
        u = torch.cat([xs[r][0][a:a + m] for r, a, m in batch])[:, :C]
        md = batch_md(batch, slots, device)
        if all(m == 1 for _, _, m in batch):
            md["cu_q"] = None
        y = ll.conv_silu(u, wt, bd, state, **md)
        at = 0
        for r, _, m in batch:
            got[r].append(y[at:at + m, :C])
            at += m

    run_portions(lens, sizes, call)
    for r in range(len(lens)):
        want = oracle.silu(oracle.causal_conv(xs[r][1], w.double(), b.double()))
        close(torch.cat(got[r]), want, TOL[dtype])
    assert taps == 1 or (state[[2, 5]] == 9).all()


# ----------------------------------------------------------------------------- recurrence
SCANS = [(4, 16, 24, 2), (2, 32, 64, 1), (3, 10, 7, 1), (2, 40, 128, 2), (4, 8, 36, 4), (1, 64, 160, 1), (2, 24, 200, 2),
         (1, 4, 300, 1), (2, 16, 30, 1), (1, 8, 250, 1)]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,P,N,G", SCANS)
@pytest.mark.parametrize("sizes", [[700], [2, 1, 3], [65, 2, 64, 1, 1, 63], [257, 8, 7, 128, 129]])
def test_recurrence_in_portions(device, dtype, H, P, N, G, sizes):
    if device == "cpu" and N > 100:
        pytest.skip("covered by the other sizes")
    lens = [530, 1, 70, 33] if device == "cuda" else [70, 1, 33]
    inner, C = H * P, H * P + 2 * G * N
    A_log, bias, D = rnd(H, seed=1), rnd(H, seed=2, scale=0.5) - 1, rnd(H, seed=3)
    dev = [t.to(device) for t in (A_log, bias, D)]
    xs = [acts(rnd(n, C, seed=20 + r, scale=0.7), dtype, device, ll.pad8(C)) for r, n in enumerate(lens)]
    dts = [acts(rnd(n, H, seed=30 + r), dtype, device, H + 3) for r, n in enumerate(lens)]
    state = torch.full((6, H, P, N), 5.0, device=device)
    slots, got = [2, 5, 0, 3], [[] for _ in lens]

    def call(batch):
        md = batch_md(batch, slots, device)
        md.pop("q_to_seq")
        if all(m == 1 for _, _, m in batch):
            md["cu_q"] = None
        x = torch.cat([xs[r][0][a:a + m] for r, a, m in batch])
        dt = torch.cat([dts[r][0][a:a + m] for r, a, m in batch])[:, :H]
        if device == "cuda" and md["cu_q"] is not None:          # the other form, on a copy of the state
            other = state.clone()
            y2 = ll.ssm_scan(x, dt, *dev, other, H=H, P=P, N=N, G=G, by_rows=True, **md)
        y = ll.ssm_scan(x, dt, *dev, state, H=H, P=P, N=N, G=G, min_q=min(m for _, _, m in batch), **md)
        if device == "cuda" and md["cu_q"] is not None:
            close(y[:, :inner], y2[:, :inner].double().cpu(), TOL[dtype])
            close(state[md["state_slots"].long()], other[md["state_slots"].long()].double().cpu(), 2e-4)
        at = 0
        for r, _, m in batch:
            got[r].append(y[at:at + m, :inner])
            at += m

    run_portions(lens, sizes, call)
    for r, n in enumerate(lens):
        x, dt = xs[r][1], torch.nn.functional.softplus(dts[r][1] + bias.double(), threshold=1e9)
        y, S = oracle.ssm_scan(x[:, :inner].view(n, H, P), x[:, inner:inner + G * N].view(n, G, N), x[:, inner + G * N:].view(n, G, N),
                               dt, A_log.double(), D.double())
        close(torch.cat(got[r]), y.reshape(n, inner), TOL[dtype])
        close(state[slots[r]], S.transpose(1, 2), 5e-5)       # the state is fp32 whatever the activations are
    assert (state[[1, 4]] == 5).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("inner,parts", [(32, 1), (48, 4), (30, 3), (2064, 2)])
def test_gate_and_grouped_norm(device, dtype, inner, parts):
    y, yd = acts(rnd(5, inner, seed=1), dtype, device, ll.pad8(inner))
    y[:, : inner // parts] *= 0.01                              # parts of different size: one common norm would show
    yd[:, : inner // parts] = y[:, : inner // parts].double().cpu()
    z, zd = acts(rnd(5, inner, seed=2), dtype, device, ll.pad8(inner) + 24)
    w = 1 + 0.2 * rnd(inner, seed=3)
    got = ll.gated_group_norm(y, z, w.to(device), parts, 1e-5)
    close(got[:, :inner], oracle.gated_group_norm(yd, zd, w.double(), parts, 1e-5), TOL[dtype])
    assert not got[:, inner:].any()

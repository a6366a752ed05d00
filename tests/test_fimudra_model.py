"""The Fimudra design through the engine - weight loading, pages and state slots, ragged and decode steps, scheduler, sampling,
trace replay - against the plain whole-sequence implementation."""
import copy
import functools
import io
import json

import pytest
import torch

import fimudra_cases as cases
import fimudra_oracle as oracle
from fimudra_cases import CONFIGS, expected
from layer_list_cases import row_errors, tokens, write_model
from omni_infer_b200.engine.engine_core import LLM, EngineConfig, EngineCore
from omni_infer_b200.engine.request import SamplingParams
from omni_infer_b200.engine.trace_replay import TraceReplay
from omni_infer_b200.models.config import ModelConfig, get_config
from test_layer_list_model import RUNS, portions, run

# Most rows / all rows / the typical row.  In 16 bits a close choice of experts may fall the other way, which moves that row and,
# through the states, a little the rows after it: only the typical rows are held to rounding there, and all rows of the
# configurations that choose every expert.  A first token may be far above the typical error in any precision: its head outputs
# are one value vector times a scalar, and the norm after them undoes a small scalar.
TOL = {"float32": (3e-5, 1e-3, 1e-5), "bfloat16": (0.12, 0.4, 0.04)}


@pytest.fixture(autouse=True)
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def build(cfg, w, device, dtype, blocks=24, block_size=64, **kw):
    mc = ModelConfig.from_hf_dict(cfg)
    mc.dtype = dtype
    kw.setdefault("max_num_seqs", 4)
    kw.setdefault("max_model_len", 512)
    return EngineCore(EngineConfig(model="x", device=device, block_size=block_size, num_kv_blocks=blocks, **kw), model_cfg=mc,
                      weights=list(w.items()))


def engine(name, device, dtype, seed=0, **kw):
    return build(CONFIGS[name], cases.weights(CONFIGS[name], seed), device, dtype, **kw)


def check(got, want, dtype, exact_choice):
    e = row_errors(got, want)
    most, every, typical = TOL[dtype]
    assert float(e.median()) < typical and float(e.quantile(0.8)) < most, (float(e.max()), float(e.median()))
    if exact_choice or dtype == "float32":
        assert float(e.max()) < every, (float(e.max()), int(e.argmax()))


def chosen(name):
    """Does every mixture of the configuration choose all of its experts?"""
    return name == "wide"


# ----------------------------------------------------------------------------- the same logits however they are computed
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", CONFIGS)
def test_cuts_of_one_sequence(name, device, dtype):
    """Whole prompt; one token at a time from the start; a prompt and long decoding; portions down to two tokens."""
    n = 150
    toks = tokens(n, CONFIGS[name]["vocab"], 1)
    eng = engine(name, device, dtype)
    for sizes in ([n], [1], [100] + [1] * 50, [2, 3], [65, 1, 64, 2], [63, 17], [16, 7, 8, 1]):
        got = run(eng, {"a": toks}, [[("a", m)] for m in portions(n, sizes)])["a"]
        check(got, expected(name, 0, toks), dtype, chosen(name))
    assert eng.kv.num_free_blocks == 23 and len(eng.kv.free_state_slots) == 4


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", CONFIGS)
def test_batches_of_unequal_requests(name, device, dtype):
    """Portions beside single tokens, requests that pause and come back, pages and slots used again; each as if it were alone."""
    V = CONFIGS[name]["vocab"]
    seqs = {"a": tokens(140, V, 1), "b": tokens(33, V, 2), "c": tokens(1, V, 3), "d": tokens(90, V, 4), "e": tokens(67, V, 5)}
    plan = [[("a", 64), ("b", 1), ("c", 1), ("d", 30)], [("b", 1), ("a", 2)], [("d", 2), ("b", 17)], [("a", 1), ("b", 1), ("d", 1), ("e", 1)],
            [("e", 3), ("b", 13), ("a", 40)], [("e", 40), ("d", 1), ("a", 3)], [("a", 1), ("d", 1), ("e", 1)], [("a", 29), ("d", 55), ("e", 1)],
            [("e", 21), ("c", 1)], [("b", 33), ("c", 1)]]
    eng = engine(name, device, dtype, blocks=10)
    got = run(eng, seqs, plan)
    for i, t in seqs.items():
        for k in range(0, len(got[i]), len(t)):
            if len(t) > 1 or dtype == "float32":
                check(got[i][k:k + len(t)], expected(name, 0, t), dtype, chosen(name))
    assert eng.kv.num_free_blocks == 9 and len(eng.kv.free_state_slots) == 4


@pytest.mark.parametrize("device,dtype", RUNS)
def test_longer_than_a_chunk_and_small_pages(device, dtype):
    """Sequences over several chunks of 128 tokens, cut at and around their edges; pages of 16 and of 128 tokens."""
    toks = tokens(330, CONFIGS["wide"]["vocab"], 7)
    for bs, sizes in ((16, [330]), (64, [128, 1, 127, 74]), (128, [129, 1, 1, 126, 73]), (64, [255, 2, 73])):
        eng = engine("wide", device, dtype, block_size=bs, blocks=24 if bs > 16 else 40)
        got = run(eng, {"a": toks}, [[("a", m)] for m in portions(330, sizes)])["a"]
        check(got, expected("wide", 0, toks), dtype, True)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("streams", [1, 2, 5])
@pytest.mark.parametrize("kind", ["wkv", "parallel"])
def test_stacks_of_one_kind(device, dtype, streams, kind):
    """Also without any page (WKV only), with one stream and with more than the specialised kernels take."""
    make = {"wkv": cases.wkv, "parallel": cases.parallel}[kind]
    cfg = cases.config([make(mlp=cases.all_of()), make(mlp=None)], streams=streams)
    w = cases.weights(cfg, 8)
    mc = ModelConfig.from_hf_dict(cfg)
    mc.dtype = dtype
    eng = EngineCore(EngineConfig(model="x", device=device, block_size=64, max_num_seqs=2, max_model_len=256), model_cfg=mc,
                     weights=list(w.items()))      # pool sized by the engine
    toks = tokens(90, 97, 3)
    got = run(eng, {"a": toks}, [[("a", m)] for m in (40, 2, 1, 1, 46)])["a"]
    check(got, oracle.forward(cfg, w, toks), dtype, True)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_residual_after_every_layer(device, dtype):
    """The sum of the streams between the layers, a looped layer counted each time."""
    name = "plain" if dtype == "float32" else "wide"
    cfg = CONFIGS[name]
    eng = engine(name, device, dtype)
    model, seen, toks = eng.worker.runner.model.model, [], tokens(23, cfg["vocab"], 2)
    from omni_infer_b200.models import layer_list as mod
    step = mod.stream_step

    def spy(x, y, *a, last=False, **k):
        h = step(x, y, *a, last=False, **k)      # the last update writes the streams back, too
        seen.append(x[:, :, :cfg["width"]].sum(1).double().cpu())
        return h

    mod.stream_step = spy
    try:
        run(eng, {"a": toks}, [[("a", len(toks))]])
    finally:
        mod.stream_step = step
    want, at = [], -1
    oracle.forward(cfg, cases.weights(cfg), toks, want)
    assert len(model.layers) == len(want)
    for L, w in zip(cfg["layers"], want):
        at += 2 if L["mlp"] else 1
        err = (seen[at] - w).pow(2).mean().sqrt() / w.pow(2).mean().sqrt()
        assert float(err) < (1e-5 if dtype == "float32" else 0.03)
    assert at == len(seen) - 1


# ----------------------------------------------------------------------------- far tokens, first tokens
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
def test_far_token_through_the_attention(device, dtype, decode):
    """Every query looks for one rare token; its place - first token, page borders, hundreds back - shows in the logits, and so
    does the sink."""
    cfg = cases.config([cases.parallel(heads=2, kv_heads=1, dim=16, vdim=16, rot=0, left_scale=3.0, right_scale=0.05, mlp=None)], width=32, vocab=16, streams=1)
    w = cases.weights(cfg, 3)
    w["embed"][:, 0], w["embed"][:, 5] = 2.0, -0.5
    w["embed"][9, 5] = 3.0
    for t, col in (("q", 0), ("k", 5)):
        w["l0.mix.left." + t].zero_()
        w["l0.mix.left." + t][:, col] = 1.4
    eng = build(cfg, w, device, dtype, blocks=8, max_num_seqs=2)
    n = 300
    base = [t % 8 for t in tokens(n, 16, 4)]
    plain = oracle.forward(cfg, w, base)[-1:]
    no_sink = dict(w, **{"l0.mix.left.sink": torch.full((2,), -30.0)})
    for at in (0, 1, 63, 64, 127, 128, 255, n - 2):
        toks = list(base)
        toks[at] = 9
        got = run(eng, {"a": toks}, [[("a", n - 1)], [("a", 1)]] if decode else [[("a", n)]])["a"]
        want = oracle.forward(cfg, w, toks)
        lim = 2e-5 if dtype == "float32" else 0.06
        assert float((row_errors(got, want)).max()) < lim
        assert float(row_errors(plain, want[-1:])[0]) > 0.2, "the case does not show the far token"
    assert float(row_errors(oracle.forward(cfg, no_sink, toks)[:2], want[:2]).max()) > 0.2, "the case does not show the sink"


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("kind", ["wkv", "memory"])
def test_far_token_lives_in_the_recurrent_state(device, dtype, kind):
    """Slow decay: what the first tokens wrote still shows hundreds of tokens later, and a fresh request in the same slot does
    not see it."""
    if kind == "wkv":
        cfg = cases.config([cases.wkv(heads=2, dim=16, mlp=None)], width=32, vocab=16, streams=2)
        w = cases.weights(cfg, 5)
        w["l0.mix.w0"].fill_(-8.0)
        w["l0.mix.w2"].mul_(0.1)
        w["l0.mix.mu.k"].zero_()
    else:
        cfg = cases.config([cases.parallel(heads=2, kv_heads=1, dim=16, vdim=16, m_heads=2, m_dim=16, m_vdim=16, cap=20.0, left_scale=0.05,
                                           mlp=None)], width=32, vocab=16, streams=2)
        w = cases.weights(cfg, 5)
        w["l0.mix.right.f.b"].fill_(12.0)
    # keys of the first tokens' kind only
    key = w["l0.mix.k" if kind == "wkv" else "l0.mix.right.k"]
    key[:, :] = key[:, 3:4] * 3 * (torch.arange(32) == 3)
    w["embed"][:, 3] = 0.0
    w["embed"][9, 3] = 6.0
    w["l0.hc1.out"].fill_(5.0)
    eng = build(cfg, w, device, dtype, blocks=10, max_num_seqs=1)
    a = [9, 3, 9, 5] * 5 + [t % 8 for t in tokens(280, 16, 1)]
    b = tokens(20, 8, 2) + a[20:]
    outs = []
    for toks in (a, b, a):
        got = run(eng, {"a": toks}, [[("a", m)] for m in [200, 64, 2] + [1] * 34])["a"]
        want = oracle.forward(cfg, w, toks)
        assert float(row_errors(got, want).max()) < (3e-5 if dtype == "float32" else 0.1)
        outs.append((got, want))
    assert float(row_errors(outs[0][1][-1:], outs[1][1][-1:])[0]) > 0.3, "the case does not show the far tokens"
    assert torch.allclose(outs[0][0], outs[2][0], atol=1e-4)


# ----------------------------------------------------------------------------- generation
@functools.lru_cache(maxsize=None)
def safe_greedy(name, prompt, n, margin):
    """Greedy continuation of the oracle, cut where the two best logits come closer than ``margin``."""
    toks, w = list(prompt), cases.weights(CONFIGS[name], 0)
    for _ in range(n):
        last = oracle.forward(CONFIGS[name], w, toks)[-1]
        top = last.topk(2).values
        if float(top[0] - top[1]) < margin * float(last.std()):
            break
        toks.append(int(last.argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("mode", ["plain", "chunked", "mixed", "preempted", "multi-step"])
def test_greedy_generation(device, dtype, mode):
    name = "plain" if dtype == "float32" else "wide"
    kw = {"plain": {}, "chunked": dict(enable_chunked_prefill=True, max_num_batched_tokens=24),
          "mixed": dict(enable_chunked_prefill=True, mixed_batches=True, max_num_batched_tokens=24),
          "preempted": dict(block_size=16, blocks=9, enable_chunked_prefill=True, mixed_batches=True, max_num_batched_tokens=40),
          "multi-step": dict(num_step=3)}[mode]
    eng = engine(name, device, dtype, **kw)
    V = CONFIGS[name]["vocab"]
    prompts = [tokens(n, V, 40 + n) for n in (1, 30, 47, 5, 19)]
    ids = [eng.add_request(p, SamplingParams(max_tokens=12, ignore_eos=True)) for p in prompts]
    outs = eng.run_until_done(2000)
    compared = 0
    for i, p in zip(ids, prompts):
        want = safe_greedy(name, tuple(p), 12, 0.002 if dtype == "float32" else 0.3)
        assert len(outs[i]) == 12 and outs[i][: len(want)] == want
        compared += len(want)
    assert compared > 8
    assert len(eng.kv.free_state_slots) == 4
    if mode == "preempted":
        assert eng.scheduler.stats["preemptions"] > 0


def test_sampling_and_llm_front_end():
    llm = LLM("tiny-fimudra", model_config=get_config("tiny-fimudra"), device="cpu", num_kv_blocks=16, block_size=16, max_model_len=128,
              max_num_seqs=2)
    outs = llm.generate([[1, 2, 3], [4] * 30], SamplingParams(max_tokens=6, temperature=0.8, top_k=20, ignore_eos=True, repetition_penalty=1.1))
    assert [len(o) for o in outs] == [6, 6] and all(0 <= t < 512 for o in outs for t in o)


# ----------------------------------------------------------------------------- configuration, loading, caches, replay
def test_configuration_reader():
    c = ModelConfig.from_hf_dict(CONFIGS["plain"])
    assert c.architecture == "Fimudra" and c.streams == 2 and c.embedding_scale == 5.0 and c.has_recurrent_state
    p = c.layers[0].parallel
    assert p.left.sink and not p.left.qk_norm and p.left.rot_scaling["factor"] == 4.0 and p.left.rot_scaling["original_max_position_embeddings"] == 128
    assert (p.left_scale, p.right_scale, p.right.gate_cap, p.right.vdim) == (0.7, 1.3, 9.0, 24)
    assert c.layers[4].weights_of == 0 and c.layers[1].wkv.heads == 3 and c.layers[3].experts.identity == 2
    e = c.layers[2].experts
    assert (e.experts, e.top, e.ff, e.limit, e.scale, e.shared_ff, e.shared_limit) == (5, 3, 24, 1.5, 1.7, 40, 0.8)
    assert c.unresolved_sizes() and not get_config("tiny-fimudra").unresolved_sizes()
    odd = ModelConfig.from_hf_dict(CONFIGS["odd"])
    assert odd.layers[1].experts is None and odd.layers[1].parallel.left.rot_dims == 0 and odd.layers[3].parallel.left.rot_scaling is None

    def bad(match, change):
        d = copy.deepcopy(CONFIGS["plain"])
        change(d)
        with pytest.raises(ValueError, match=match):
            ModelConfig.from_hf_dict(d)

    bad("share weights", lambda d: d["layers"][4]["mixer"].update(left_scale=0.2))
    bad("takes its weights", lambda d: d["layers"][4].update(weights_of=4))
    bad("takes its weights", lambda d: d["layers"][4].update(weights_of=9))
    bad("unknown mixer", lambda d: d["layers"][1].update(type="something"))
    bad("experts", lambda d: d["layers"][2]["mlp"]["router"].update(top=8))
    bad("residual", lambda d: d.pop("streams"))


def test_loader_wants_every_tensor_and_no_other():
    cfg = CONFIGS["plain"]
    w = cases.weights(cfg)
    small = dict(device="cpu", dtype="float32", blocks=4, max_model_len=64, max_num_seqs=1)
    eng = build(cfg, w, **small)
    model = eng.worker.runner.model
    # every checkpoint value arrives in exactly one place
    stored = {k: (p.data[r0:r0 + rows] if cols is None else p.data[r0:r0 + rows, :cols]) for k, (p, r0, rows, cols) in model.checkpoint_targets().items()}
    assert set(stored) == set(w) and all(torch.equal(stored[k].float(), w[k].float()) for k in w)
    assert model.model.layers[4] is model.model.layers[0]
    with pytest.raises(KeyError, match="lacks"):
        build(cfg, {k: v for k, v in w.items() if k != "l1.mix.u"}, **small)
    with pytest.raises(KeyError, match="lacks"):
        build(cfg, {k: v for k, v in w.items() if k != "l3.mix.w1"}, **small)
    with pytest.raises(KeyError, match="no parameter"):
        build(cfg, dict(w, **{"l4.norm1": w["l0.norm1"]}), **small)
    with pytest.raises(ValueError, match="shape"):
        build(cfg, dict(w, **{"l0.hc1.mix": w["l0.hc1.mix"][:1]}), **small)


def test_every_layer_run_has_a_cache_of_its_own():
    eng = engine("plain", "cpu", "float32")
    c = eng.worker.runner.kv_caches
    (k0, v0), (S0, m0) = c[0]
    (k4, v4), (S4, m4) = c[4]
    assert k0 is not k4 and S0 is not S4 and k0.shape == k4.shape == (24, 64, 2, 24) and v0.shape == (24, 64, 2, 16)
    assert S0.shape == (4, 3, 25, 16) and m0.shape == (4, 3) and S0.dtype == m0.dtype == torch.float32
    h, S = c[1]
    assert h.shape == (4, 48) and S.shape == (4, 3, 16, 16) and S.dtype == torch.float32
    m = eng.worker.runner.model
    assert m.num_kv_layers == 3 and m.kv_bytes_per_token() == 3 * 2 * (24 + 16) * 4
    flat = [t for x in c for t in (x[1] if isinstance(x[0], tuple) else x)]
    assert m.state_bytes(4) == sum(t.numel() * t.element_size() for t in flat)


def test_what_the_model_does_not_combine_with():
    for kw in (dict(enable_prefix_caching=True), dict(num_speculative_tokens=1), dict(enable_omni_attn=True, omni_attn_config={"sink": 1, "recent": 1})):
        with pytest.raises(ValueError):
            engine("plain", "cpu", "float32", **kw)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_trace_runner_on_a_model_folder(device, dtype, tmp_path):
    """The folder's tensors give the sizes that the configuration leaves open."""
    from omni_infer_b200.cli.trace_run import build_engine, replay
    name = "wide"
    cfg = CONFIGS[name]
    write_model(tmp_path, cfg, cases.weights(cfg))
    seqs = {"p": tokens(70, cfg["vocab"], 1), "q": tokens(20, cfg["vocab"], 2)}
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": seqs["p"][:50], "want": [49, 0]}, {"id": "q", "tokens": seqs["q"][:1], "want": []}],
              "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": seqs["p"][50:51], "want": [0]}, {"id": "q", "tokens": seqs["q"][1:2], "want": [0]}]},
             {"step": 2, "entries": [{"id": "q", "tokens": seqs["q"][2:], "want": []}], "end": ["q"]},
             {"step": 3, "entries": [{"id": "p", "tokens": seqs["p"][51:], "want": [18]}], "end": ["p"]}]
    eng = build_engine(str(tmp_path), dtype, 192, device=device)
    assert eng.model_cfg.layers[0].wkv.rank == cases.RANK
    done = []
    replay(eng, io.StringIO("\n".join(json.dumps(s) for s in steps)), str(tmp_path), done.append)
    assert done == [0, 1, 2, 3] and not (tmp_path / "2.f32").exists()

    def rows(k):
        return torch.frombuffer(bytearray((tmp_path / f"{k}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])

    p, q = expected(name, 0, seqs["p"]), expected(name, 0, seqs["q"])
    for got, want in ((rows(0), p[[49, 0]]), (rows(1), torch.stack([p[50], q[1]])), (rows(3), p[[69]])):
        assert float(row_errors(got, want).max()) < TOL[dtype][1] * 1.5
    with pytest.raises(RuntimeError):
        TraceReplay(eng).step([{"id": "s", "tokens": [1] * 500, "want": []}])


def test_kernel_build_takes_the_architecture_sources_only():
    from omni_infer_b200 import build as b
    _, every = b._kernel_inputs()
    _, some = b._kernel_inputs(b.ARCH_KERNELS["Fimudra"])
    assert {s.stem for s in some} == set(b.ARCH_KERNELS["Fimudra"]) < {s.stem for s in every}

"""Layer-list models through the engine - weight loading, pages and state slots, ragged and decode steps, scheduler,
sampling, trace replay - against the plain whole-sequence implementation."""
import copy
import io
import json

import pytest
import torch

import layer_list_cases as cases
import layer_list_oracle as oracle
from layer_list_cases import CONFIGS, error, expected, row_errors, tokens
from omni_infer_b200.engine.engine_core import LLM, EngineConfig, EngineCore
from omni_infer_b200.engine.kv_manager import KVCacheManager
from omni_infer_b200.engine.request import Request, SamplingParams
from omni_infer_b200.engine.trace_replay import TraceReplay
from omni_infer_b200.models.config import ModelConfig, get_config

RUNS = [pytest.param("cpu", "float32", id="cpu-float32"), pytest.param("cuda", "float32", id="cuda-float32", marks=pytest.mark.gpu),
        pytest.param("cuda", "bfloat16", id="cuda-bfloat16", marks=pytest.mark.gpu)]
# largest row error, typical row error.  Rounding to bf16 alone (the CPU references) gives 0.06 and 0.015 here.
TOL = {"float32": 2e-5, "bfloat16": 0.15}
TYPICAL = {"float32": 1e-5, "bfloat16": 0.03}
ONE_LAYER = {"float32": 1e-5, "bfloat16": 0.1}      # largest row again, rounding alone gives up to 0.05


@pytest.fixture(autouse=True)
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def engine(name, device, dtype, seed=0, blocks=24, block_size=64, **kw):
    cfg = CONFIGS[name]
    mc = ModelConfig.from_hf_dict(cfg)
    mc.dtype = dtype
    kw.setdefault("max_num_seqs", 4)
    kw.setdefault("max_model_len", 512)
    return EngineCore(EngineConfig(model=name, device=device, block_size=block_size, num_kv_blocks=blocks, **kw), model_cfg=mc,
                      weights=list(cases.weights(cfg, seed).items()))


def run(eng, seqs, plan):
    """Feeds ``seqs`` {id: tokens} by ``plan`` [[(id, count)]]; returns {id: logits of every position}.  A request ends with
    its last token; an id whose tokens are used up may start again (its pages and slot come back from the pool)."""
    tr, at, got = TraceReplay(eng), {i: 0 for i in seqs}, {i: [] for i in seqs}
    for step in plan:
        entries, end = [], []
        for i, n in step:
            a = at[i]
            entries.append({"id": i, "tokens": seqs[i][a:a + n], "want": list(range(n))})
            at[i] = a + n
            if at[i] == len(seqs[i]):
                end.append(i)
                at[i] = 0
        out = tr.step(entries, end)
        k = 0
        for i, n in step:
            got[i].append(out[k:k + n])
            k += n
    assert not tr.live
    return {i: torch.cat(v) for i, v in got.items()}


def portions(n, sizes):
    out, a, k = [], 0, 0
    while a < n:
        out.append(min(sizes[k % len(sizes)], n - a))
        a, k = a + out[-1], k + 1
    return out


def check(name, got, toks, dtype, seed=0):
    e = row_errors(got, expected(name, seed, toks))
    assert float(e.max()) < TOL[dtype] and float(e.median()) < TYPICAL[dtype], (float(e.max()), float(e.median()))


# ----------------------------------------------------------------------------- the same logits however they are computed
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", CONFIGS)
def test_cuts_of_one_sequence(name, device, dtype):
    """Whole prompt; one token at a time from the start; a prompt and long decoding; portions down to two tokens."""
    n = 150
    toks = tokens(n, CONFIGS[name]["vocab"], 1)
    eng = engine(name, device, dtype)
    for sizes in ([n], [1], [100] + [1] * 50, [2, 3], [65, 1, 64, 2], [63, 17]):
        got = run(eng, {"a": toks}, [[("a", m)] for m in portions(n, sizes)])["a"]
        check(name, got, toks, dtype)
    assert eng.kv.num_free_blocks == 23 and len(eng.kv.free_state_slots) == 4


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", CONFIGS)
def test_batches_of_unequal_requests(name, device, dtype):
    """Portions beside single tokens, requests that pause and come back, pages and slots used again."""
    V = CONFIGS[name]["vocab"]
    seqs = {"a": tokens(140, V, 1), "b": tokens(33, V, 2), "c": tokens(1, V, 3), "d": tokens(90, V, 4), "e": tokens(67, V, 5)}
    plan = [[("a", 64), ("b", 1), ("c", 1), ("d", 30)], [("b", 1), ("a", 2)], [("d", 2), ("b", 17)], [("a", 1), ("b", 1), ("d", 1), ("e", 1)],
            [("e", 3), ("b", 13), ("a", 40)], [("e", 40), ("d", 1), ("a", 3)], [("a", 1), ("d", 1), ("e", 1)], [("a", 29), ("d", 55), ("e", 1)],
            [("e", 21), ("c", 1)], [("b", 33), ("c", 1)]]
    eng = engine(name, device, dtype, blocks=10)
    got = run(eng, seqs, plan)
    check(name, got["a"], seqs["a"], dtype)
    for i in ("b", "d", "e", "c"):
        t = seqs[i]
        for k in range(0, len(got[i]), len(t)):
            check(name, got[i][k:k + len(t)], t, dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_small_pages_and_wide_pages(device, dtype):
    toks = tokens(100, CONFIGS["plain"]["vocab"], 7)
    for bs in (16, 128):
        eng = engine("plain", device, dtype, block_size=bs)
        got = run(eng, {"a": toks}, [[("a", m)] for m in portions(100, [37, 1, 1, 30])])["a"]
        check("plain", got, toks, dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("layers", [[cases.attention(ff=0), cases.attention(kv_from=0, window=9, ff=24)],
                                    [cases.mamba(ff=24), cases.mamba(groups=1, conv=2)]], ids=["attention-only", "mamba-only"])
def test_stacks_of_one_kind(device, dtype, layers):
    cfg = cases.config(layers)
    w = cases.weights(cfg, 8)
    mc = ModelConfig.from_hf_dict(cfg)
    mc.dtype = dtype
    eng = EngineCore(EngineConfig(model="x", device=device, block_size=64, max_num_seqs=2, max_model_len=256), model_cfg=mc,
                     weights=list(w.items()))      # pool sized by the engine
    toks = tokens(90, 97, 3)
    got = run(eng, {"a": toks}, [[("a", m)] for m in (40, 2, 1, 1, 46)])["a"]
    e = row_errors(got, oracle.forward(cfg, w, toks))
    assert float(e.max()) < TOL[dtype] and float(e.median()) < TYPICAL[dtype]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
def test_token_inside_and_outside_the_window_through_the_model(device, dtype, decode):
    """One attention layer whose queries look for one rare token: the logits follow it to the last place of the window and
    forget it one place further."""
    window = 20
    cfg = cases.config([cases.attention(heads=2, kv_heads=1, dim=16, vdim=16, window=window, rot=0, ff=0)], width=32, vocab=16)
    w = cases.weights(cfg, 3)
    # every query is the same vector; the rare token's key points along it, every other key the opposite way
    w["embed"][:, 0], w["embed"][:, 5] = 2.0, -0.5
    w["embed"][9, 5] = 3.0
    for t, col in (("q", 0), ("k", 5)):
        w["l0.mix." + t].zero_()
        w["l0.mix." + t][:, col] = 1.0
        w[f"l0.mix.{t}.norm"].fill_(1.0)
    mc = ModelConfig.from_hf_dict(cfg)
    mc.dtype = dtype
    eng = EngineCore(EngineConfig(model="x", device=device, block_size=64, num_kv_blocks=6, max_num_seqs=2, max_model_len=128),
                     model_cfg=mc, weights=list(w.items()))
    base = [t % 8 for t in tokens(70, 16, 4)]
    last = []
    for dist in (window - 1, window):
        toks = list(base)
        toks[69 - dist] = 9
        plan = [[("a", 69)], [("a", 1)]] if decode else [[("a", 70)]]
        got = run(eng, {"a": toks}, plan)["a"]
        want = oracle.forward(cfg, w, toks)
        assert error(got, want) < ONE_LAYER[dtype]
        last.append(want[-1])
    assert error(last[0][None], last[1][None]) > 3 * ONE_LAYER["bfloat16"], "the case does not show the edge"


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_token_lives_in_the_recurrent_state(device, dtype):
    """Slow decay: what the first tokens wrote into the state still shows hundreds of tokens later, and a fresh request in
    the same slot does not see it."""
    cfg = cases.config([cases.mamba(heads=2, vdim=16, state=16, groups=1, conv=3, norm_groups=1)], width=32, vocab=16)
    w = cases.weights(cfg, 5)
    w["l0.mix.A_log"].fill_(-7.0)
    w["l0.mix.dt_bias"].fill_(-2.0)
    w["embed"][9] *= 6
    mc = ModelConfig.from_hf_dict(cfg)
    mc.dtype = dtype
    eng = EngineCore(EngineConfig(model="x", device=device, block_size=64, num_kv_blocks=10, max_num_seqs=1, max_model_len=512),
                     model_cfg=mc, weights=list(w.items()))
    a = [9] * 20 + [t % 8 for t in tokens(280, 16, 1)]      # the first tokens write far more than the others
    b = tokens(20, 8, 2) + a[20:]
    outs = []
    for toks in (a, b, a):
        got = run(eng, {"a": toks}, [[("a", m)] for m in [200, 64, 2] + [1] * 34])["a"]
        want = oracle.forward(cfg, w, toks)
        assert error(got, want) < ONE_LAYER[dtype]
        outs.append((got, want))
    assert error(outs[0][1][-1:], outs[1][1][-1:]) > 3 * ONE_LAYER["bfloat16"], "the case does not show the far tokens"
    assert torch.allclose(outs[0][0], outs[2][0], atol=1e-5)


# ----------------------------------------------------------------------------- generation
def safe_greedy(name, prompt, n, margin):
    """Greedy continuation of the oracle, cut where the two best logits come closer than ``margin``."""
    toks = list(prompt)
    w = cases.weights(CONFIGS[name], 0)
    for _ in range(n):
        top = oracle.forward(CONFIGS[name], w, toks)[-1].topk(2).values
        if float(top[0] - top[1]) < margin:
            break
        toks.append(int(oracle.forward(CONFIGS[name], w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("mode", ["plain", "chunked", "mixed", "preempted", "multi-step"])
def test_greedy_generation(device, dtype, mode):
    name = "plain"
    kw = {"plain": {}, "chunked": dict(enable_chunked_prefill=True, max_num_batched_tokens=24),
          "mixed": dict(enable_chunked_prefill=True, mixed_batches=True, max_num_batched_tokens=24),
          "preempted": dict(block_size=16, blocks=9, enable_chunked_prefill=True, mixed_batches=True, max_num_batched_tokens=40),
          "multi-step": dict(num_step=3)}[mode]
    eng = engine(name, device, dtype, **kw)
    prompts = [tokens(n, 97, 40 + n) for n in (1, 30, 47, 5, 19)]
    ids = [eng.add_request(p, SamplingParams(max_tokens=12, ignore_eos=True)) for p in prompts]
    outs = eng.run_until_done(2000)
    compared = 0
    for i, p in zip(ids, prompts):
        want = safe_greedy(name, p, 12, 0.002 if dtype == "float32" else 0.15)
        assert len(outs[i]) == 12 and outs[i][: len(want)] == want
        compared += len(want)
    assert compared > 8
    assert len(eng.kv.free_state_slots) == 4
    if mode == "preempted":
        assert eng.scheduler.stats["preemptions"] > 0


def test_mixed_steps_carry_decoding_requests():
    eng = engine("plain", "cpu", "float32", enable_chunked_prefill=True, mixed_batches=True, max_num_batched_tokens=20)
    sp = SamplingParams(max_tokens=20, ignore_eos=True)
    eng.add_request(tokens(10, 97, 1), sp, request_id="a")
    eng.step()
    eng.add_request(tokens(50, 97, 2), sp, request_id="b")
    so = eng.scheduler.schedule()
    assert so.is_prefill and [(s.request.request_id, s.num_scheduled_tokens) for s in so.scheduled] == [("a", 1), ("b", 19)]
    eng.scheduler.update_from_output(so, eng.worker.execute_model(so))
    assert len(eng.scheduler.requests["a"].output_token_ids) == 2 and not eng.scheduler.requests["b"].output_token_ids
    with pytest.raises(ValueError):
        engine("plain", "cpu", "float32", mixed_batches=True)


def test_sampling_and_llm_front_end():
    mc = get_config("tiny-forovik")
    llm = LLM("tiny-forovik", model_config=mc, device="cpu", num_kv_blocks=16, block_size=16, max_model_len=128, max_num_seqs=2)
    outs = llm.generate([[1, 2, 3], [4] * 30], SamplingParams(max_tokens=6, temperature=0.8, top_k=20, ignore_eos=True, repetition_penalty=1.1))
    assert [len(o) for o in outs] == [6, 6] and all(0 <= t < 512 for o in outs for t in o)


# ----------------------------------------------------------------------------- configuration, loading, slots, replay
def test_configuration_reader():
    c = ModelConfig.from_hf_dict(CONFIGS["plain"])
    assert c.architecture == "Forovik" and c.vocab_size == 97 and c.hidden_size == 48 and c.rms_norm_eps == 1e-5
    assert c.has_recurrent_state and not get_config("qwen2-small").has_recurrent_state
    assert c.layers[3].attention.kv_from == 0 and c.layers[3].attention.window == 33 and c.layers[0].attention.rot_factor == 2.0
    assert c.layers[2].mamba2.groups == 3 and c.layers[2].ff == 0 and c.layers[0].ff == 40
    bad = copy.deepcopy(CONFIGS["plain"])
    bad["layers"][3]["mixer"]["kv_from"] = 1
    with pytest.raises(ValueError, match="takes its keys"):
        ModelConfig.from_hf_dict(bad)
    bad["layers"][3]["mixer"].update(kv_from=0, dim=8)
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(bad)
    bad = copy.deepcopy(CONFIGS["plain"])
    bad["layers"][1]["type"] = "something"
    with pytest.raises(ValueError, match="unknown mixer"):
        ModelConfig.from_hf_dict(bad)
    bad = copy.deepcopy(CONFIGS["plain"])
    bad["layers"][0]["mlp"]["kind"] = "moe"
    with pytest.raises(ValueError, match="feed-forward"):
        ModelConfig.from_hf_dict(bad)


def test_loader_wants_every_tensor_and_no_other():
    cfg = CONFIGS["plain"]
    w = cases.weights(cfg)

    def build(weights):
        mc = ModelConfig.from_hf_dict(cfg)
        mc.dtype = "float32"
        return EngineCore(EngineConfig(model="x", device="cpu", num_kv_blocks=4, max_model_len=64, max_num_seqs=1), model_cfg=mc,
                          weights=list(weights.items()))

    build(w)
    with pytest.raises(KeyError, match="lacks"):
        build({k: v for k, v in w.items() if k != "l1.mix.D"})
    with pytest.raises(KeyError, match="no parameter"):
        build(dict(w, extra=w["embed"]))
    with pytest.raises(ValueError, match="shape"):
        build(dict(w, embed=w["embed"][:, :-1]))


def test_shared_keys_share_one_cache():
    eng = engine("plain", "cpu", "float32")
    c = eng.worker.runner.kv_caches
    assert c[3][0] is c[0][0] and c[3][1] is c[0][1]
    assert c[0][0].shape == (24, 64, 2, 24) and c[0][1].shape == (24, 64, 2, 16)
    assert c[1][1].shape == (4, 4, 16, 24) and c[1][1].dtype == torch.float32 and c[1][0].shape == (4, 3, 160)


def test_state_slots_follow_the_pages():
    kv = KVCacheManager(9, 16, num_state_slots=2)
    a, b, c = (Request(i, [0] * 20) for i in "abc")
    assert kv.allocate_slots(a, 20) is not None and kv.allocate_slots(b, 20) is not None
    assert {a.state_slot, b.state_slot} == {0, 1}
    assert kv.allocate_slots(c, 20) is None and c.state_slot == -1 and not c.block_ids     # pages are there, slots are not
    slot = a.state_slot
    kv.free(a)
    kv.free(a)
    assert a.state_slot == -1 and kv.allocate_slots(c, 20) is not None and c.state_slot == slot
    with pytest.raises(ValueError, match="prefix caching"):
        KVCacheManager(9, 16, enable_prefix_caching=True, num_state_slots=2)


def test_what_the_model_does_not_combine_with():
    with pytest.raises(ValueError):
        engine("plain", "cpu", "float32", enable_prefix_caching=True)
    with pytest.raises(ValueError):
        engine("plain", "cpu", "float32", num_speculative_tokens=1)
    with pytest.raises(ValueError):
        engine("plain", "cpu", "float32", enable_omni_attn=True, omni_attn_config={"sink": 1, "recent": 1})


@pytest.mark.parametrize("device,dtype", RUNS)
def test_trace_runner_on_a_model_folder(device, dtype, tmp_path):
    from omni_infer_b200.cli.trace_run import build_engine, replay
    name = "odd"
    cfg = CONFIGS[name]
    cases.write_model(tmp_path, cfg, cases.weights(cfg))
    seqs = {"p": tokens(70, cfg["vocab"], 1), "q": tokens(20, cfg["vocab"], 2)}
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": seqs["p"][:50], "want": [49, 0]}, {"id": "q", "tokens": seqs["q"][:1], "want": []}],
              "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": seqs["p"][50:51], "want": [0]}, {"id": "q", "tokens": seqs["q"][1:2], "want": [0]}]},
             {"step": 2, "entries": [{"id": "q", "tokens": seqs["q"][2:], "want": []}], "end": ["q"]},
             {"step": 3, "entries": [{"id": "p", "tokens": seqs["p"][51:], "want": [18]}], "end": ["p"]}]
    eng = build_engine(str(tmp_path), dtype, 192, device=device)
    assert eng.kv.num_free_blocks == 3
    done = []
    replay(eng, io.StringIO("\n".join(json.dumps(s) for s in steps)), str(tmp_path), done.append)
    assert done == [0, 1, 2, 3] and not (tmp_path / "2.f32").exists()
    V = cfg["vocab"]

    def rows(k):
        return torch.frombuffer(bytearray((tmp_path / f"{k}.f32").read_bytes()), dtype=torch.float32).view(-1, V)

    p, q = expected(name, 0, seqs["p"]), expected(name, 0, seqs["q"])
    for got, want in ((rows(0), p[[49, 0]]), (rows(1), torch.stack([p[50], q[1]])), (rows(3), p[[69]])):
        assert error(got, want) < TOL[dtype] * 1.5
    assert eng.kv.num_free_blocks == 3
    tr = TraceReplay(eng)
    with pytest.raises(ValueError):
        tr.step([{"id": "r", "tokens": [V], "want": []}])
    with pytest.raises(ValueError):
        tr.step([{"id": "r", "tokens": [1, 2], "want": [2]}])
    with pytest.raises(RuntimeError):
        tr.step([{"id": "s", "tokens": [1] * 500, "want": []}])


def test_kernel_build_takes_the_architecture_sources_only(monkeypatch, tmp_path):
    from omni_infer_b200 import build
    _, every = build._kernel_inputs()
    _, some = build._kernel_inputs(build.ARCH_KERNELS["Forovik"])
    assert {s.stem for s in some} == set(build.ARCH_KERNELS["Forovik"]) < {s.stem for s in every}

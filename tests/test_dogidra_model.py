"""Dogidra through the engine against the plain implementation: whole prompts, portions, decoding, mixed batches, pages
and slots used again, greedy generation through `generate`, `serve` and a session; on CPU in fp32, on the GPU in fp32 and bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dogidra_oracle as oracle  # noqa: E402
from dogidra_util import CONFIGS, TOL, case_for, checkpoint, config, engine, mixer, run_portions, tokens  # noqa: E402
from zml_b200 import safetensors  # noqa: E402
from zml_b200.models import hub  # noqa: E402
from zml_b200.models.common import SamplingStrategy, detect_model_type  # noqa: E402
from zml_b200.models.dogidra import DogidraConfig, DogidraModel  # noqa: E402
from zml_b200.serving.engine import OutOfPages, Session  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TARGETS = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
           pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]
_oracle_cache = {}


@pytest.fixture(scope="module")
def repos(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            path = tmp_path_factory.mktemp(name)
            made[name] = (path,) + checkpoint(str(path), name, seed=sorted(CONFIGS).index(name))
        return made[name]
    return get


def expected(repos, name, n, seed):
    key = (name, n, seed)
    if key not in _oracle_cache:
        _, cfg, w = repos(name)
        t = tokens(cfg, n, seed)
        _oracle_cache[key] = (t, oracle.forward(cfg, w, t))
    return _oracle_cache[key]


def row_errors(got, want):
    """Root mean square of every row's difference over that of the expected rows, means taken off."""
    off = lambda x: x - x.mean(-1, keepdims=True)
    return np.sqrt((off(got - want) ** 2).mean(-1)) / np.sqrt((off(want) ** 2).mean())


def check(got, want, dtype, what=""):
    e = row_errors(np.asarray(got, dtype=np.float64), want)
    over = np.nonzero(e > TOL[dtype])[0]
    assert len(over) == 0 and np.median(e) < TOL[dtype] / 2, (what, len(over), over[:5], e[over[:5]], e.max(), np.median(e))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", [n for n in sorted(CONFIGS) if "," not in n])
def test_whole_decode_and_portions_agree_with_the_oracle(repos, name, target):
    device, dtype = target
    name = case_for(name, dtype)
    path, _, _ = repos(name)
    toks, want = expected(repos, name, 150, 1)
    eng = engine(path, device, dtype, max_tokens=192)
    for sizes in ([150], [110, 1], [2, 3, 61, 5, 2, 64, 1]):       # whole; prefill then decode; portions over page borders
        check(run_portions(eng, toks, sizes), want, dtype, (name, sizes))


@pytest.mark.parametrize("target", TARGETS[:2])
@pytest.mark.parametrize("name", ["mixed", "ones", "odd", "wide", "heads"])
def test_stream_behind_every_run_of_a_layer(repos, name, target):
    device, dtype = target
    path, cfg, w = repos(name)
    toks, layers = tokens(cfg, 90, 7), []
    oracle.forward(cfg, w, toks, layers)
    assert len(layers) == len(oracle.runs(cfg))
    eng = engine(path, device, dtype, max_tokens=128)
    r = eng.open_request()
    eng.append_tokens(r, toks)
    ids, meta = eng._varlen_meta([(r, 0, len(toks))], [], None)
    for got, want in zip(eng.model.layer_steps(ids, meta, eng.kv_cache), layers, strict=True):
        err = np.abs(got.double().cpu().numpy() - want)
        assert err.max() < 3e-4 * np.abs(want).max()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_token_by_token_from_the_first_one(repos, name, target):
    device, dtype = target
    name = case_for(name, dtype)
    path, _, _ = repos(name)
    toks, want = expected(repos, name, 80, 2)
    eng = engine(path, device, dtype, max_tokens=128)
    check(run_portions(eng, toks, [1]), want, dtype)
    check(run_portions(eng, toks, [2]), want, dtype)               # the same pages again


@pytest.mark.parametrize("target", TARGETS)
def test_mixed_batches_equal_each_request_alone(repos, target):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, end and hand on pages and slots."""
    device, dtype = target
    name = case_for("mixed", dtype)
    path, cfg, _ = repos(name)
    reqs = {i: expected(repos, name, n, 10 + i) for i, n in enumerate((131, 40, 1, 97, 70, 3))}
    eng = engine(path, device, dtype, max_tokens=384, slots=3)
    rng = np.random.default_rng(5)
    live, at, got, waiting, pages0 = {}, {}, {i: [] for i in reqs}, list(reqs), eng.pool.num_free
    steps = 0
    while waiting or live:
        while waiting and len(live) < 3:
            i = waiting.pop(0)
            live[i], at[i] = eng.open_request(), 0
        chosen = [i for i in live if rng.random() < 0.8] or list(live)
        entries, ns = [], []
        for i in chosen:
            left = len(reqs[i][0]) - at[i]
            n = int(min(left, 1 if (steps % 4 == 3 or rng.random() < 0.4) else rng.integers(2, 40)))
            entries.append((live[i], reqs[i][0][at[i]:at[i] + n]))
            ns.append(n)
        lg = eng.step(entries, [list(range(n)) for n in ns]).float().cpu().numpy()
        base = 0
        for i, n in zip(chosen, ns):
            got[i].append(lg[base:base + n])
            base += n
            at[i] += n
            if at[i] == len(reqs[i][0]):
                eng.release(live.pop(i))
        steps += 1
    assert eng.pool.num_free == pages0 and len(eng.slot_free) == 3
    for i in reqs:
        check(np.concatenate(got[i]), reqs[i][1], dtype, i)


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding_passes_windows_blocks_and_pages(repos, target):
    device, dtype = target
    name = case_for("mixed", dtype)
    path, _, _ = repos(name)
    toks, want = expected(repos, name, 300, 3)
    eng = engine(path, device, dtype, max_tokens=320)
    check(run_portions(eng, toks, [5, 1]), want, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_captured_and_eager_decode_steps_agree(repos, dtype):
    path, _, _ = repos("wide")
    toks, _ = expected(repos, "wide", 150, 1)
    a, b = (run_portions(engine(path, "cuda", dtype, max_tokens=192, use_graphs=g), toks, [100, 1]) for g in (True, False))
    assert np.array_equal(a, b)


@pytest.mark.parametrize("target", TARGETS)
def test_only_wanted_logits_come_back(repos, target):
    device, dtype = target
    path, _, _ = repos("mixed")
    toks, want = expected(repos, "mixed", 80, 2)
    eng = engine(path, device, dtype, max_tokens=192)
    a, b = eng.open_request(), eng.open_request()
    assert eng.step([(a, toks[:10]), (b, toks[:30])]) is None
    lg = eng.step([(a, toks[10:40]), (b, toks[30:31])], [[0, 29, 3], [0]]).float().cpu().numpy()
    assert lg.shape[0] == 4
    lg2 = eng.step([(a, toks[40:41]), (b, toks[31:32])], [[], [0]]).float().cpu().numpy()
    assert lg2.shape[0] == 1
    got, rows = np.concatenate([lg, lg2]), want[[10, 39, 13, 30, 31]]
    assert np.median(row_errors(got.astype(np.float64), rows)) < TOL[dtype]
    if dtype == torch.float32:
        check(got, rows, dtype)


# ------------------------------------------------------------------ generation
@pytest.mark.parametrize("target", TARGETS[:2])
def test_greedy_generation_through_engine_serve_and_session(repos, target):
    device, dtype = target
    path, cfg, w = repos("mixed")
    prompts = [tokens(cfg, n, 20 + n) for n in (1, 2, 63, 64, 30)]
    want = [oracle.greedy(cfg, w, p, 6) for p in prompts]
    eng = engine(path, device, dtype, max_tokens=640, max_batch=5)
    outs, stats = eng.generate(prompts, 6)
    assert outs == want and stats.output_tokens == 30
    eng = engine(path, device, dtype, max_tokens=256, max_batch=2, max_prefill_tokens=17)      # rows and pages go round
    outs, _ = eng.serve(prompts, 6, sync_interval=2)
    assert outs == want
    s = Session(eng, 128)
    s.run_prefill(prompts[4][:11])
    s.run_prefill(prompts[4][11:])
    assert s.run_decode(max_new_tokens=6) == want[4]
    s.close()


@pytest.mark.gpu
def test_bf16_generation_with_graphs_equals_the_eager_loop(repos):
    path, cfg, _ = repos("wide")
    prompts = [tokens(cfg, n, 40 + n) for n in (3, 90, 20)]
    a, _ = engine(path, "cuda", torch.bfloat16, max_tokens=640).generate(prompts, 12)
    b, _ = engine(path, "cuda", torch.bfloat16, max_tokens=640, use_graphs=False).generate(prompts, 12)
    assert a == b
    eng = engine(path, "cuda", torch.bfloat16, max_tokens=640)
    c, _ = eng.generate(prompts, 12, SamplingStrategy(topk=4, temperature=0.7), seed=3)
    assert c == eng.generate(prompts, 12, SamplingStrategy(topk=4, temperature=0.7), seed=3)[0]


# ------------------------------------------------------------------ configuration, checkpoint, command line
def test_config_registry_and_errors():
    cfg = CONFIGS["mixed"]
    assert detect_model_type(cfg) == "dogidra"
    c = DogidraConfig.from_hf(cfg)
    assert c.to_json() == cfg and c.hidden_size == 96
    for name in ("wide", "odd", "ones"):
        assert DogidraConfig.from_hf(CONFIGS[name]).to_json() == CONFIGS[name]
    left = lambda d: d["layers"][0]["mixer"]["left"]
    for breakage in (lambda d: d["layers"][0].update(type="mamba"), lambda d: d["layers"][0]["mlp"].update(kind="dense"),
                     lambda d: d["layers"][0]["mlp"]["router"].update(top=7), lambda d: d.pop("embedding"), lambda d: d["canon"].update(taps=9),
                     lambda d: d["canon"].update(taps=0), lambda d: left(d)["mask"].update(size=0), lambda d: d["loop"].update(stop=5),
                     lambda d: d["loop"].update(start=3), lambda d: d["loop"].update(times=0)):
        d = json.loads(json.dumps(cfg))
        breakage(d)
        with pytest.raises(ValueError):
            DogidraConfig.from_hf(d)


def test_runs_of_a_loop():
    c = DogidraConfig.from_hf(CONFIGS["mixed"])
    assert c.runs() == [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)] == oracle.runs(CONFIGS["mixed"])
    assert DogidraConfig.from_hf(CONFIGS["ones"]).runs() == [(0, True)]
    assert DogidraConfig.from_hf(CONFIGS["odd"]).runs() == [(0, False), (1, False)]
    assert DogidraConfig.from_hf(CONFIGS["wide"]).runs() == [(0, True), (1, False), (2, False)] * 2


@pytest.mark.parametrize("bad", [mixer(heads=3, kv_heads=2), mixer(rot=5), mixer(rot=26), mixer(pool=-1)])
def test_sizes_that_no_kernel_takes_are_refused_at_load(bad):
    with pytest.raises(ValueError):
        DogidraModel(DogidraConfig.from_hf(config([(bad, None)])), device="cpu", dtype=torch.float32).init_random(0)


def test_taps_of_the_checkpoint_must_fit():
    cfg = config([(mixer(), None)])
    shapes = DogidraConfig.from_hf(cfg).checkpoint_shapes()

    class Store:
        def load_tensor(self, name, device=None, dtype=None, rows=None, cols=None):
            w = torch.zeros(shapes[name] if "canon" not in name else (96, 4), dtype=dtype)
            return w[slice(*(rows or (None, None)))][..., slice(*(cols or (None, None)))]
    with pytest.raises(ValueError, match="taps"):
        DogidraModel(DogidraConfig.from_hf(cfg), device="cpu", dtype=torch.float32).load(Store())


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_checkpoint_round_trip(repos, name):
    path, cfg, w = repos(name)
    model, tok = hub.load_model(str(path), device="cpu", dtype=torch.float32)
    assert tok is None and model.weight_bytes() > 0
    sd = model.state_dict_hf()
    assert set(sd) == set(w) and all(np.array_equal(sd[k].double().numpy(), w[k].reshape(sd[k].shape)) for k in w)
    assert {k: tuple(v.shape) for k, v in sd.items()} == {k: tuple(v) for k, v in model.checkpoint_shapes().items()}
    assert sum(v.numel() for v in sd.values()) == DogidraConfig.from_hf(cfg).num_params()


def test_every_pass_has_caches_and_states_of_its_own(repos):
    path, _, _ = repos("mixed")
    model, _ = hub.load_model(str(path), device="cpu", dtype=torch.float32)
    kv = model.alloc_kv_cache(3, 64)
    model.alloc_state(2)
    assert len(kv) == len(model.runs) == 8 and len({t.data_ptr() for c in kv for t in c}) == 4 * 8
    states = [t for r in model.runs for t in r.states()]
    assert len({t.data_ptr() for t in states}) == len(states)
    assert model.runs[1].layer is model.runs[3].layer and model.state_bytes_per_slot() == sum(t[0].numel() * 4 for t in states)
    assert [tuple(t.shape[:2]) for t in kv[0]] == [(3, 64), (3, 64), (3, 13), (3, 13)]


def test_pages_and_slots_run_out_and_come_back(repos):
    path, cfg, _ = repos("mixed")
    eng = engine(path, "cpu", torch.float32, max_tokens=128, slots=2)
    a, b = eng.open_request(), eng.open_request()
    with pytest.raises(OutOfPages):
        eng.open_request()
    eng.step([(a, tokens(cfg, 65, 1))])
    with pytest.raises(OutOfPages):
        eng.step([(b, tokens(cfg, 1, 1))])
    eng.release(a)
    eng.step([(b, tokens(cfg, 1, 1))])
    eng.open_request()


@pytest.mark.parametrize("target", TARGETS)
def test_trace_run_program(repos, target, tmp_path):
    device, dtype = target
    path, _, _ = repos("mixed")
    toks, want = expected(repos, "mixed", 80, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:50], "want": [49, 0]}, {"id": "b", "tokens": toks[:1], "want": []}], "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[50:51], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[51:52], "want": [0]}, {"id": "c", "tokens": toks[:2], "want": [1]}], "end": ["a", "c"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(path), "--dtype", "float32" if dtype == torch.float32 else "bfloat16",
                        "--out", str(tmp_path), "--max-tokens", "256", "--device", device], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32"]
    got = np.concatenate([np.fromfile(tmp_path / f, "<f4").reshape(-1, want.shape[1]) for f in ("0.f32", "2.f32")])
    assert np.median(row_errors(got.astype(np.float64), want[[49, 0, 51, 1]])) < TOL[dtype]


def test_llm_command_line(repos):
    path, cfg, w = repos("ones")
    want = oracle.greedy(cfg, w, [3, 9, 27], 4)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "examples", "llm", "main.py"), f"--model={path}", "--prompt=3 9 27", "--seqlen=64",
                        "--max-new-tokens=4", "--cpu"], capture_output=True, text=True, timeout=180)
    assert r.returncode == 0, r.stderr[-2000:]
    assert " ".join(map(str, want)) in r.stdout

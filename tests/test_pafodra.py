"""Pafodra through the framework's model, state manager and generation, against the plain statement of the design."""
import json
import os
import subprocess
import sys

import pytest
import torch

import pafodra_models as pm
import plain_pafodra as plain

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]


def _device(name):
    if name == "cuda":
        if not torch.cuda.is_available():
            pytest.skip("no GPU")
        from easyllm_b200.ops import cuda
        cuda.lib()
    return torch.device(name)


@pytest.fixture(autouse=True)
def _few_threads():
    """The plain statement runs on tiny tensors: threads only get in its way."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


_cache = {}


@pytest.fixture
def models(tmp_path_factory):
    def get(name, device, dtype=torch.float32):
        """(cfg, weights, model on the device); the weights are exact in bf16, so both dtypes hold the same ones."""
        key = (name, device.type, dtype)
        if key not in _cache:
            from easyllm_b200.models.hf_models import CausalLM
            cfg = pm.CONFIGS[name]
            w = pm.weights(cfg, seed=len(name), bf16=True)
            path = pm.save(tmp_path_factory.mktemp(name), cfg, w)
            _cache[key] = cfg, w, CausalLM.from_pretrained(path, torch_dtype=dtype).to(device).eval()
        return _cache[key]
    return get


_want = {}


def oracle(name, cfg, w, toks):
    key = (name, tuple(toks))
    if key not in _want:
        _want[key] = plain.forward(cfg, w, toks)
    return _want[key]


def error(got, want, dtype=torch.float32):
    """Root mean square difference of a row of logits over their spread: the largest of all rows in fp32; in bf16 the
    upper quartile, because rounding can turn a close choice of experts into the other one and its rows stand out."""
    d = got.detach().double().cpu() - want
    rows = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float(rows.max() if dtype == torch.float32 else rows.quantile(0.75))


LIMIT = {torch.float32: 3e-5, torch.bfloat16: 0.06}


def run(model, state, slots, parts):
    h, meta = model.step(state, slots, parts)
    return [x for x in model.logits(h).split([len(p) for p in parts])]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", list(pm.CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_prompt_and_first_tokens(models, name, device, dtype):
    dev = _device(device)
    cfg, w, model = models(name, dev, dtype)
    for n in (1, 2, 70):
        toks = pm.tokens(cfg, n)
        state = model.new_state(1, 16)
        got = run(model, state, [state.open()], [toks])[0]
        assert error(got, oracle(name, cfg, w, toks), dtype) < LIMIT[dtype], (n, dtype)
        with torch.no_grad():                 # the call without a state is the same model
            full = model(input_ids=torch.tensor([toks], device=dev))["logits"][0]
        assert error(full, oracle(name, cfg, w, toks), dtype) < LIMIT[dtype], (n, dtype)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", list(pm.CONFIGS))
def test_residual_stream_after_every_layer(models, name, device):
    dev = _device(device)
    cfg, w, model = models(name, dev)
    toks, trace, mine = pm.tokens(cfg, 19, 5), [], []
    plain.forward(cfg, w, toks, trace=trace)
    hooks = [l.register_forward_hook(lambda m, a, out: mine.append(out[0].double().cpu())) for l in {*model.model.layers}]
    try:
        state = model.new_state(1, 16)
        run(model, state, [state.open()], [toks])
    finally:
        for h in hooks:
            h.remove()
    assert len(mine) == len(trace) == len(cfg["layers"])
    for got, want in zip(mine, trace):
        assert (got - want).abs().max() < 2e-5 * want.abs().max()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", list(pm.CONFIGS))
@pytest.mark.parametrize("cut", [1, 2, 3, 16, 17, 33])
def test_portions_of_a_prompt_then_decoding(models, name, device, cut):
    """However a sequence is cut into steps (down to single tokens), the logits are those of the whole."""
    dev = _device(device)
    cfg, w, model = models(name, dev)
    toks = pm.tokens(cfg, 70)
    state = model.new_state(1, 16)
    slot, got = state.open(), []
    for a in range(0, 64, cut):
        got.append(run(model, state, [slot], [toks[a:min(a + cut, 64)]])[0])
    for t in toks[64:]:
        got.append(run(model, state, [slot], [[t]])[0])
    assert error(torch.cat(got), oracle(name, cfg, w, toks)) < LIMIT[torch.float32]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_unequal_batch_ends_and_slots_used_again(models, name, device, dtype):
    """Requests of unequal length prefill and decode as one batch, shorter ones end earlier, and the next batch gets
    their slots: everything equals each request alone."""
    dev = _device(device)
    cfg, w, model = models(name, dev, dtype)
    state = model.new_state(2, 16)
    for batch in range(3):
        reqs = [pm.tokens(cfg, n, 10 * batch + i) for i, n in enumerate([(9, 40, 23), (33, 5), (2, 61, 31, 20)][batch])]
        slots = [state.open() for _ in reqs]
        got = [[x] for x in run(model, state, slots, [r[:-(len(r) // 2)] for r in reqs])]
        at = [len(r) - len(r) // 2 for r in reqs]
        while True:
            live = [i for i, r in enumerate(reqs) if at[i] < len(r)]
            if not live:
                break
            outs = run(model, state, [slots[i] for i in live], [[reqs[i][at[i]]] for i in live])
            for i, o in zip(live, outs):
                got[i].append(o)
                at[i] += 1
                if at[i] == len(reqs[i]):
                    state.close(slots[i])
        for r, o in zip(reqs, got):
            assert error(torch.cat(o), oracle(name, cfg, w, r), dtype) < LIMIT[dtype], (batch, len(r))
    assert sorted(state.free) == list(range(state.slots)) and state.slots == 4


@pytest.mark.parametrize("device", DEVICES)
def test_prompts_and_decoding_tokens_in_one_step(models, device):
    """A step may bring a new prompt, a continued prompt and single tokens at once."""
    dev = _device(device)
    cfg, w, model = models("aligned", dev)
    a, b, c = (pm.tokens(cfg, n, 30 + n) for n in (50, 44, 30))
    state = model.new_state(3, 16)
    sa, sb, sc = (state.open() for _ in range(3))
    ga, gb = ([x] for x in run(model, state, [sa, sb], [a[:49], b[:20]]))
    ya, yb, gc = run(model, state, [sa, sb, sc], [a[49:], b[20:], c])
    for got, toks in ((torch.cat(ga + [ya]), a), (torch.cat(gb + [yb]), b), (gc, c)):
        assert error(got, oracle("aligned", cfg, w, toks)) < LIMIT[torch.float32]


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding_over_the_growth_of_the_cache(models, device):
    """Decoding far past the first block of cache positions equals one long prompt, also for the request beside it."""
    dev = _device(device)
    cfg, w, model = models("odd", dev)
    a, b = pm.tokens(cfg, 540, 7), pm.tokens(cfg, 300, 8)
    whole = []
    for t in (a, b):
        s = model.new_state(1, 600)
        whole.append(run(model, s, [s.open()], [t])[0])
    state = model.new_state(2, 32)
    sa, sb = state.open(), state.open()
    ga, gb = ([x] for x in run(model, state, [sa, sb], [a[:250], b[:10]]))
    for i in range(290):
        xa, xb = run(model, state, [sa, sb], [[a[250 + i]], [b[10 + i]]])
        ga.append(xa), gb.append(xb)
    assert state.capacity >= 540
    for got, want in ((torch.cat(ga), whole[0]), (torch.cat(gb), whole[1])):
        assert error(got, want.double().cpu()) < LIMIT[torch.float32]
    assert error(whole[1][:90], oracle("odd", cfg, w, b[:90])) < LIMIT[torch.float32]


def _greedy_oracle(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(plain.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_of_an_unequal_batch(models, device):
    dev = _device(device)
    cfg, w, model = models("odd", dev)
    prompts, n = [pm.tokens(cfg, k, 50 + k) for k in (5, 11, 1)], 8
    want = [_greedy_oracle(cfg, w, p, n) for p in prompts]
    s = max(map(len, prompts))
    for left in (True, False):
        ids = torch.zeros(3, s, dtype=torch.long)
        mask = torch.zeros_like(ids)
        for i, p in enumerate(prompts):
            at = slice(s - len(p), s) if left else slice(0, len(p))
            ids[i, at], mask[i, at] = torch.tensor(p), 1
        out = model.generate(ids.to(dev), attention_mask=mask.to(dev), max_new_tokens=n)
        assert out[:, s:].tolist() == want
    stream = [int(t[0]) for t in model.generate_stream(torch.tensor([prompts[1]], device=dev), max_new_tokens=n)]
    assert stream == want[1]
    # an end token stops its row, the others go on and the row is filled
    eos = want[1][3]
    out = model.generate(ids.to(dev), attention_mask=mask.to(dev), max_new_tokens=n, eos_token_id=eos)[:, s:].tolist()
    for row, full in zip(out, want):
        cut = full.index(eos) + 1 if eos in full else len(full)
        assert row[:cut] == full[:cut] and all(t == eos for t in row[cut:])


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["aligned", "wide"])
def test_replayed_decode_steps_equal_eager_ones(models, name):
    """The decode step as a CUDA graph, over the border of a cache tile, for an unequal batch."""
    dev = _device("cuda")
    cfg, w, model = models(name, dev, torch.bfloat16)
    from easyllm_b200.models.hf_models.state import DecodeGraph
    reqs = [pm.tokens(cfg, 90, 1), pm.tokens(cfg, 40, 2)]
    logits = []
    for replay in (False, True):
        state = model.new_state(2, 128)
        slots = [state.open(), state.open()]
        run(model, state, slots, [r[:-35] for r in reqs])
        graph, got = None, []
        for i in range(35):
            ids = torch.tensor([r[-35 + i] for r in reqs], device=dev)
            if graph is not None:
                got.append(graph.step(ids).clone())
            else:
                got.append(model.logits(model.step(state, slots, ids)[0]))
                graph = DecodeGraph(model, state, slots) if replay else None
        assert state.lengths[:2] == [90, 40] or state.lengths[slots[0]] == 90
        logits.append(torch.stack(got))
    assert error(logits[1].flatten(0, 1), logits[0].flatten(0, 1).double().cpu(), torch.bfloat16) < 1e-3


def test_text_generation_entry_point(models):
    """The inference loop of the HF runner on a model from the registry."""
    from easyllm_b200.config.registry import MODULE_ZOO_REGISTRY
    from easyllm_b200.data import SimpleTokenizer
    from easyllm_b200.infer.hf_inference import generate_text
    torch.manual_seed(0)
    cfg = dict(pm.CONFIGS["odd"], vocab=300)
    model = MODULE_ZOO_REGISTRY.build({"type": "PafodraForCausalLM", "kwargs": {"arch": cfg}}).eval()
    tok = SimpleTokenizer(vocab_size=300)
    ids = tok("hello")["input_ids"]
    text = generate_text(model, tok, ids, torch.device("cpu"), {"max_new_tokens": 5})
    out = model.generate(torch.tensor([ids]), max_new_tokens=5, eos_token_id=tok.eos_token_id)[0, len(ids):].tolist()
    assert text == tok.decode([t for t in out if t != tok.eos_token_id])
    sampled = model.generate(torch.tensor([ids]), max_new_tokens=5, do_sample=True, top_k=5, repetition_penalty=1.2)
    assert sampled.shape[1] == len(ids) + 5
    with pytest.raises(NotImplementedError):
        model(input_ids=torch.tensor([ids]), labels=torch.tensor([ids]))


def test_checkpoint_round_trip_and_registry(models, tmp_path):
    from easyllm_b200.config.registry import MODULE_ZOO_REGISTRY
    cfg, w, model = models("aligned", torch.device("cpu"))
    layers = model.model.layers
    assert layers[3] is layers[0] and layers[5] is layers[1] and layers[4].mlp is None
    model.save_pretrained(str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    sd = torch.load(tmp_path / "pytorch_model.bin")
    assert set(sd) == set(w) and all(torch.equal(sd[n].float(), w[n].float()) for n in w)
    again = MODULE_ZOO_REGISTRY.build({"type": "AutoCausalLM", "kwargs": {"model_name_or_path": str(tmp_path)}}).eval()
    toks = torch.tensor([pm.tokens(cfg, 12)])
    with torch.no_grad():
        assert torch.equal(again(input_ids=toks)["logits"], model(input_ids=toks)["logits"])


def test_bad_configs_are_refused():
    from easyllm_b200.models.hf_models import arch_from_hf_config
    base = pm.CONFIGS["odd"]

    def broken(i, **kw):
        layers = [dict(l) for l in base["layers"]]
        layers[i].update(kw)
        return dict(base, layers=layers)
    for cfg in (broken(0, type="mystery"), broken(1, mixer=dict(heads=5, kv_heads=2, dim=12, vdim=18, scale=0.4)),
                broken(1, mixer=dict(heads=5, kv_heads=1, dim=12, vdim=18)), broken(1, mlp=dict(kind="cubic", ff=4)),
                broken(3, weights_of=9)):
        with pytest.raises(ValueError):
            arch_from_hf_config(cfg)


@pytest.mark.parametrize("device", DEVICES)
def test_trace_replay(models, tmp_path, device):
    """bin/trace_run: two requests as one batch, then decoded; the logits asked for, and nothing else."""
    _device(device)
    cfg = pm.CONFIGS["odd"]
    w = pm.weights(cfg, seed=3, bf16=True)
    path = pm.save(tmp_path / "m", cfg, w)
    a, b = pm.tokens(cfg, 12, 1), pm.tokens(cfg, 7, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:10], "want": [0, 9]}, {"id": "b", "tokens": b[:6], "want": [3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[6:], "want": []}, {"id": "a", "tokens": a[10:11], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[11:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "19", "--device", device], input="\n".join(map(json.dumps, steps)) + "\n",
                       capture_output=True, text=True, timeout=300, env=dict(os.environ, PATH=os.path.dirname(sys.executable)
                                                                             + os.pathsep + os.environ["PATH"]))
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]

    def read(n):
        return torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    wa, wb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    assert error(read(0), torch.stack([wa[0], wa[9], wb[3]])) < 3e-5
    assert error(read(2), wa[11:]) < 3e-5

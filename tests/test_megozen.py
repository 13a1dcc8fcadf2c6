"""Megozen through the framework's model, state manager and generation, against the plain statement of the design."""
import json
import os
import subprocess
import sys

import pytest
import torch

import megozen_models as mm
import plain_megozen as plain
from test_pafodra import DEVICES, ROOT, _device, _few_threads, error, run  # noqa: F401

F32, BF16 = torch.float32, torch.bfloat16
LIMIT = {F32: 3e-5, BF16: 0.06}
_cache, _want = {}, {}


@pytest.fixture
def models(tmp_path_factory):
    def get(name, device, dtype=F32):
        """(cfg, weights, model on the device); the weights are exact in bf16, so both dtypes hold the same ones."""
        key = (name, device.type, dtype)
        if key not in _cache:
            from easyllm_b200.models.hf_models import CausalLM
            cfg = mm.CONFIGS[name]
            w = mm.weights(cfg, seed=len(name), bf16=True)
            path = mm.save(tmp_path_factory.mktemp(name), cfg, w)
            _cache[key] = cfg, w, CausalLM.from_pretrained(path, torch_dtype=dtype).to(device).eval()
        return _cache[key]
    return get


def oracle(name, cfg, w, toks):
    key = (name, tuple(toks))
    if key not in _want:
        _want[key] = plain.forward(cfg, w, toks)
    return _want[key]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", list(mm.CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_whole_prompt_and_first_tokens(models, name, device, dtype):
    dev = _device(device)
    cfg, w, model = models(name, dev, dtype)
    for n in (1, 2, 3, 70):
        toks = mm.tokens(cfg, n)
        state = model.new_state(1, 16)
        got = run(model, state, [state.open()], [toks])[0]
        assert error(got, oracle(name, cfg, w, toks), dtype) < LIMIT[dtype], (n, dtype)
        with torch.no_grad():                 # the call without a state is the same model
            full = model(input_ids=torch.tensor([toks], device=dev))["logits"][0]
        assert error(full, oracle(name, cfg, w, toks), dtype) < LIMIT[dtype], (n, dtype)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompt_over_many_tiles_then_decoding(models, device, dtype):
    """A prompt far past every window, the two ways through the latent side by side: whole, and its last tokens decoded."""
    dev = _device(device)
    cfg, w, model = models("aligned", dev, dtype)
    toks = mm.tokens(cfg, 300, 4)
    want = oracle("aligned", cfg, w, toks)
    state = model.new_state(2, 16)
    slot = state.open()
    got = run(model, state, [slot], [toks])[0]
    assert error(got, want, dtype) < LIMIT[dtype]
    state.close(slot)
    slot, got = state.open(), []
    got.append(run(model, state, [slot], [toks[:250]])[0])
    for t in toks[250:]:
        got.append(run(model, state, [slot], [[t]])[0])
    assert error(torch.cat(got), want, dtype) < LIMIT[dtype]
    with torch.no_grad():                     # packed documents without a state
        ids = torch.tensor([toks[:170] + toks[:130]], device=dev)
        out = model(input_ids=ids, cu_seqlens=torch.tensor([0, 170, 300], dtype=torch.int32))["logits"][0]
    assert error(out[:170], want[:170], dtype) < LIMIT[dtype] and error(out[170:], want[:130], dtype) < LIMIT[dtype]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", list(mm.CONFIGS))
def test_residual_stream_after_every_layer(models, name, device):
    dev = _device(device)
    cfg, w, model = models(name, dev)
    toks, trace, mine = mm.tokens(cfg, 23, 5), [], []
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
@pytest.mark.parametrize("name", list(mm.CONFIGS))
@pytest.mark.parametrize("cut", [1, 2, 3, 17, 33])
def test_portions_of_a_prompt_then_decoding(models, name, device, cut):
    """However a sequence is cut into steps (down to single tokens), the logits are those of the whole."""
    dev = _device(device)
    cfg, w, model = models(name, dev)
    toks = mm.tokens(cfg, 70)
    state = model.new_state(1, 16)
    slot, got = state.open(), []
    for a in range(0, 64, cut):
        got.append(run(model, state, [slot], [toks[a:min(a + cut, 64)]])[0])
    for t in toks[64:]:
        got.append(run(model, state, [slot], [[t]])[0])
    assert error(torch.cat(got), oracle(name, cfg, w, toks)) < LIMIT[F32]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_unequal_batch_ends_and_slots_used_again(models, name, device, dtype):
    """Requests of unequal length prefill and decode as one batch, shorter ones end earlier, and the next batch gets
    their slots: everything equals each request alone."""
    dev = _device(device)
    cfg, w, model = models(name, dev, dtype)
    state = model.new_state(2, 16)
    for batch in range(3):
        reqs = [mm.tokens(cfg, n, 10 * batch + i) for i, n in enumerate([(9, 40, 23), (33, 5), (2, 61, 31, 20)][batch])]
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
    a, b, c = (mm.tokens(cfg, n, 30 + n) for n in (50, 44, 30))
    state = model.new_state(3, 16)
    sa, sb, sc = (state.open() for _ in range(3))
    ga, gb = ([x] for x in run(model, state, [sa, sb], [a[:49], b[:20]]))
    ya, yb, gc = run(model, state, [sa, sb, sc], [a[49:], b[20:], c])
    for got, toks in ((torch.cat(ga + [ya]), a), (torch.cat(gb + [yb]), b), (gc, c)):
        assert error(got, oracle("aligned", cfg, w, toks)) < LIMIT[F32]


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding_over_the_growth_of_the_cache(models, device):
    """Decoding far past the first block of cache positions equals one long prompt, also for the request beside it."""
    dev = _device(device)
    cfg, w, model = models("odd", dev)
    a, b = mm.tokens(cfg, 540, 7), mm.tokens(cfg, 300, 8)
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
        assert error(got, want.double().cpu()) < LIMIT[F32]
    assert error(whole[1][:90], oracle("odd", cfg, w, b[:90])) < LIMIT[F32]


@pytest.mark.parametrize("device", DEVICES)
def test_far_key_decides_and_the_window_hides_it(models, device):
    """A layer whose queries look for one token: changing that token changes the logits as long as it is in sight of the
    window, in a prompt and in decoding, and not by a bit once it is one token too far."""
    dev = _device(device)
    W = 21
    cfg = mm.config(40, 32, [mm.lat(2, 16, 8, 16, 16, 1.0, W, mlp=None)], 3, 1, 1)
    w = mm.weights(cfg, 3)
    from easyllm_b200.models.hf_models import CausalLM
    from easyllm_b200.models.hf_models.io import import_state
    from easyllm_b200.models.hf_models.modeling import arch_from_hf_config
    model = CausalLM(arch_from_hf_config(cfg)).eval()
    model.load_state_dict(import_state(w, model.arch))
    model = model.to(dev)
    toks = mm.tokens(cfg, 60, 9)
    far = 30                                  # pairs: tokens 30 and 31 change, so positions 30 + W and on do not see them
    other = toks[:far] + [(toks[far] + 1) % 40] + toks[far + 1:]

    def logits(t, cut):
        state = model.new_state(1, 16)
        slot = state.open()
        out = [run(model, state, [slot], [t[:cut]])[0]] if cut else []
        return torch.cat(out + [run(model, state, [slot], [[x]])[0] for x in t[cut:]])
    for cut in (60, 33, 0):
        x, y = logits(toks, cut), logits(other, cut)
        same = (x - y).abs().amax(-1) == 0
        assert same[:far].all() and same[far + 1 + W:].all()
        # token far + 1 (its pair changed) is still in sight at far + W, out of sight one later
        assert not same[[far, far + 1, far + W - 1, far + W]].any()
        assert error(x, plain.forward(cfg, w, toks)) < LIMIT[F32]


def _greedy_oracle(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(plain.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_of_an_unequal_batch(models, device):
    dev = _device(device)
    cfg, w, model = models("odd", dev)
    prompts, n = [mm.tokens(cfg, k, 50 + k) for k in (5, 11, 1)], 8
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


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["aligned", "wide", "odd"])
def test_replayed_decode_steps_equal_eager_ones(models, name):
    """The decode step as a CUDA graph, over the border of a cache tile and of the windows, for an unequal batch."""
    dev = _device("cuda")
    cfg, w, model = models(name, dev, BF16)
    from easyllm_b200.models.hf_models.state import DecodeGraph
    reqs = [mm.tokens(cfg, 90, 1), mm.tokens(cfg, 40, 2)]
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
        logits.append(torch.stack(got))
    assert error(logits[1].flatten(0, 1), logits[0].flatten(0, 1).double().cpu(), BF16) < 2e-2


def test_text_generation_entry_point():
    """The inference loop of the HF runner on a model from the registry; what an inference-only family refuses."""
    from easyllm_b200.config.registry import MODULE_ZOO_REGISTRY
    from easyllm_b200.models import hf_models  # noqa: F401  (fills the registry)
    from easyllm_b200.data import SimpleTokenizer
    from easyllm_b200.infer.hf_inference import generate_text
    torch.manual_seed(0)
    cfg = dict(mm.CONFIGS["odd"], vocab=300)
    model = MODULE_ZOO_REGISTRY.build({"type": "MegozenForCausalLM", "kwargs": {"arch": cfg}}).eval()
    tok = SimpleTokenizer(vocab_size=300)
    ids = tok("hello")["input_ids"]
    text = generate_text(model, tok, ids, torch.device("cpu"), {"max_new_tokens": 5})
    out = model.generate(torch.tensor([ids]), max_new_tokens=5, eos_token_id=tok.eos_token_id)[0, len(ids):].tolist()
    assert text == tok.decode([t for t in out if t != tok.eos_token_id])
    sampled = model.generate(torch.tensor([ids]), max_new_tokens=5, do_sample=True, top_k=5, repetition_penalty=1.2)
    assert sampled.shape[1] == len(ids) + 5
    with pytest.raises(NotImplementedError):
        model(input_ids=torch.tensor([ids]), labels=torch.tensor([ids]))
    with pytest.raises(NotImplementedError):          # the embedding looks at token pairs: there are no ids to look at
        model.generate(torch.tensor([ids]), max_new_tokens=2, soft_prefix={"embeds": torch.zeros(3, cfg["width"])})


def test_checkpoint_round_trip_and_registry(models, tmp_path):
    from easyllm_b200.config.registry import MODULE_ZOO_REGISTRY
    cfg, w, model = models("aligned", torch.device("cpu"))
    layers = model.model.layers
    assert layers[3] is layers[0] and layers[2].mlp is None
    model.save_pretrained(str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    sd = torch.load(tmp_path / "pytorch_model.bin")
    assert set(sd) == set(w) and all(torch.equal(sd[n].float(), w[n].float()) for n in w)
    again = MODULE_ZOO_REGISTRY.build({"type": "AutoCausalLM", "kwargs": {"model_name_or_path": str(tmp_path)}}).eval()
    toks = torch.tensor([mm.tokens(cfg, 12)])
    with torch.no_grad():
        assert torch.equal(again(input_ids=toks)["logits"], model(input_ids=toks)["logits"])


def test_changed_weights_reach_the_derived_ones(models):
    """The transposed key product is made anew when its weight changes."""
    cfg, w, _ = models("odd", torch.device("cpu"))
    from easyllm_b200.models.hf_models import CausalLM
    from easyllm_b200.models.hf_models.io import import_state
    from easyllm_b200.models.hf_models.modeling import arch_from_hf_config
    model = CausalLM(arch_from_hf_config(cfg)).eval()
    toks = mm.tokens(cfg, 9)
    for seed in (1, 2):
        w = mm.weights(cfg, seed)
        model.load_state_dict(import_state(w, model.arch))
        state = model.new_state(1, 16)
        assert error(run(model, state, [state.open()], [toks])[0], plain.forward(cfg, w, toks)) < LIMIT[F32]


def test_bad_configs_are_refused():
    from easyllm_b200.models.hf_models import arch_from_hf_config
    base = mm.CONFIGS["odd"]

    def broken(i, mixer=None, **kw):
        layers = [dict(l) for l in base["layers"]]
        layers[i].update(kw)
        layers[i]["mixer"] = dict(layers[i]["mixer"], **(mixer or {}))
        return dict(base, layers=layers)
    short = broken(0)
    del short["layers"][0]["mixer"]["kv_rank"]
    for cfg in (broken(0, type="attention"), broken(1, mlp=dict(kind="dense", ff=4)), broken(2, weights_of=9), short,
                broken(0, mixer=dict(rot=mm.rot(8))), broken(0, mixer=dict(rot=mm.rot(3))), broken(1, mixer=dict(mask=dict(size=0)))):
        with pytest.raises(ValueError):
            arch_from_hf_config(cfg)


@pytest.mark.parametrize("device", DEVICES)
def test_trace_replay(tmp_path, device):
    """bin/trace_run: two requests as one batch, then decoded; the logits asked for, and nothing else."""
    _device(device)
    cfg = mm.CONFIGS["odd"]
    w = mm.weights(cfg, seed=3, bf16=True)
    path = mm.save(tmp_path / "m", cfg, w)
    a, b = mm.tokens(cfg, 12, 1), mm.tokens(cfg, 7, 2)
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
        return torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=F32).view(-1, cfg["vocab"])
    wa, wb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    assert error(read(0), torch.stack([wa[0], wa[9], wb[3]])) < 3e-5
    assert error(read(2), wa[11:]) < 3e-5

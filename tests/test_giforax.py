"""Giforax through the framework's engine (config reader, loader, cache and state managers, batch layout, kernels) against the
plain double-precision implementation of ``giforax_oracle.py``. Every case runs on the CPU path in fp32 and, on a GPU, in true
fp32 and in bf16. The mechanisms alone are compared on the CPU here and kernel by kernel in ``test_giforax_ops_gpu.py``."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import giforax_oracle as oracle
from hybrid_testing import (LIMIT, WHERE, Replay, check, engine, error, gpu, in_portions, one_thread,
                            tokens_of, unequal_requests)
from test_netezen import one_sequence
from tokenweave_b200 import LLM, SamplingParams
from tokenweave_b200.config import EngineArgs, ModelConfig
from tokenweave_b200.layers.mixers import GroupedAttention, rope_table
from tokenweave_b200.ops import hybrid as hops
from tokenweave_b200.ops import reference

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CPU = ("cpu", "float32")


@pytest.fixture(autouse=True)
def _one_thread():
    yield from one_thread()


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(name, where) -> (config, weights, folder), each made once. In bf16 hardly a choice of experts hangs on a rounding."""
    made = {}

    def get(name, where=CPU):
        key = (name, where[1] == "bfloat16")
        if key not in made:
            cfg = oracle.CONFIGS[name]
            w = oracle.random_weights(cfg, seed=len(name), decided=key[1])
            made[key] = (cfg, w, oracle.save(cfg, w, tmp_path_factory.mktemp(name)))
        return made[key]
    return get


@pytest.fixture(scope="module")
def expected(models):
    """Oracle logits of a model's token sequences, each computed once."""
    made = {}

    def get(name, where, tokens):
        key = (name, where[1] == "bfloat16", tuple(tokens))
        if key not in made:
            cfg, w, _ = models(name, where)
            made[key] = oracle.logits(cfg, w, tokens)
        return made[key]
    return get


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", oracle.CONFIGS)
def test_whole_prompts(models, expected, name, where):
    cfg, w, path = models(name, where)
    with Replay(path, where, blocks=20) as r:
        for n in (1, 2, 15, 64, 290):
            t = tokens_of(cfg, n, n)
            check(r.step([("a", t, range(n))], ["a"]), expected(name, where, t), where, f"{n} tokens")


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", oracle.CONFIGS)
def test_portions_and_single_tokens(models, expected, name, where):
    """However a prompt is cut - token by token, in twos, across pages, tiles and chunks - every position comes out alike."""
    cfg, w, path = models(name, where)
    t = tokens_of(cfg, 190, 3)
    with Replay(path, where, blocks=13) as r:
        for portions in ([1], [2], [3, 2, 70, 2, 16, 17, 33], [64], [100, 1], [130, 2, 1]):
            check(in_portions(r, "a", t, portions), expected(name, where, t), where, str(portions))


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["aligned", "odd", "recurrent"])
def test_unequal_requests_share_steps_pages_and_slots(models, name, where):
    cfg, w, path = models(name, where)
    unequal_requests(oracle, cfg, w, path, where)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["aligned", "recurrent"])
def test_long_decoding(models, expected, name, where):
    """Chunks begin and end among decoded tokens many times; states are carried through hundreds of steps."""
    cfg, w, path = models(name, where)
    t = tokens_of(cfg, 420, 8)
    with Replay(path, where, blocks=28) as r:
        check(in_portions(r, "a", t, [20, 1]), expected(name, where, t), where)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("page", [16, 64, 128])
def test_page_sizes(models, expected, where, page):
    cfg, w, path = models("odd", where)
    t = tokens_of(cfg, 250, 9)
    with Replay(path, where, blocks=256 // page, page=page) as r:
        check(in_portions(r, "a", t, [page - 1, 2, page, 1, 1, 40]), expected("odd", where, t), where)


@pytest.mark.parametrize("name", oracle.CONFIGS)
def test_the_residual_stream_after_every_layer(models, monkeypatch, name):
    cfg, w, path = models(name)
    t, got, want = tokens_of(cfg, 40, 2), [], []
    oracle.logits(cfg, w, t, want)
    plain = hops.sandwich_step

    def spy(y, x32, post, nxt, eps, xa, coef=None, results=None, last=False):
        plain(y, x32, post, nxt, eps, xa, coef, results, last)
        if coef is not None:
            got.append(x32[:, :cfg["width"]].clone())
    monkeypatch.setattr(hops, "sandwich_step", spy)
    with Replay(path, CPU, blocks=4) as r:
        r.step([("a", t, [])], ["a"])
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        assert (a - b.float()).abs().max() < 1e-4


# ---- chunks, far keys, states ----------------------------------------------------------------------------------------------
def stand_out(cfg, weights, tokens, key, query):
    """Edits the first layer so that the score of (query, key) in its last head stands out, rotated as they are: the query's
    projection gets a large component along the key, and other keys hardly count."""
    w, m, eps = {k: v.double() for k, v in weights.items()}, cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    h = oracle.layer_norm(x, w["l0.norm1"], w["l0.norm1.b"], eps)
    G, D, V = m["kv_heads"], m["dim"], m["vdim"]
    k = (h @ w["l0.mix.k"].T).view(len(tokens), G, D)[key, G - 1]
    along = oracle.rotate(k.view(1, 1, -1), m["rot"], [key - query]).view(-1)
    q, o = w["l0.mix.q"].clone(), w["l0.mix.o"].clone()
    q[-D:] += 200.0 / (along @ along).sqrt() * torch.outer(along, h[query] / (h[query] @ h[query]))
    o[:, -V:] *= 8                                    # the head carries the layer's output
    pb = torch.full_like(weights["l0.mix.pb"], -8.0)
    return {**weights, "l0.mix.q": q.to(torch.bfloat16), "l0.mix.o": o.to(torch.bfloat16), "l0.mix.pb": pb}


LAST = 330                                            # the asking position


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("chunk,key,seen", [
    (16, 320, True), (16, 319, False), (64, 320, True), (64, 319, False), (100, 300, True), (100, 299, False),
    (127, 254, True), (127, 253, False), (128, 256, True), (128, 255, False), (129, 258, True), (129, 257, False),
    (165, 330, True), (165, 329, False), (166, 166, True), (166, 165, False), (200, 200, True), (200, 199, False),
    (331, 0, True), (5000, 0, True), (330, 329, False), (1, 330, True), (1, 329, False), (2, 330, True), (3, 330, True),
    (3, 329, False), (329, 329, True), (329, 328, False)])
def test_a_position_sees_its_chunk(tmp_path, monkeypatch, where, chunk, key, seen):
    """The last position asks for one key - in a prompt, in portions and decoded. A key it sees decides the answer; one that
    it does not see would, were the chunk's edge one token off."""
    n = LAST + 1
    cfg = oracle.model([oracle.attn_layer(4, 2, 64, 40, 32, chunk, None, scale=0.25)], width=80)
    t = [x % 90 for x in tokens_of(cfg, n, 21)]
    t[key], t[-1] = 95, 96                            # two tokens that occur once
    if key == LAST:
        t[-1] = 95
    w = stand_out(cfg, oracle.random_weights(cfg, 4), t, key, LAST)
    want = oracle.logits(cfg, w, t)[-1:]
    assert oracle.visible(LAST, key, chunk) == seen
    plain = oracle.visible
    monkeypatch.setattr(oracle, "visible", lambda i, j, c: plain(i, j, c) != (i == LAST and j == key))
    assert error(oracle.logits(cfg, w, t)[-1:].float(), want)[0] > 2 * LIMIT["bfloat16"]
    path = oracle.save(cfg, w, tmp_path)
    with Replay(path, where, blocks=(n + 63) // 64, page=64) as r:
        check(r.step([("a", t, [n - 1])], ["a"]), want, where, "prompt")
        r.step([("b", t[:n // 2], [])])
        r.step([("b", t[n // 2:-1], [])])
        check(r.step([("b", t[-1:], [0])], ["b"]), want, where, "decoded")
        check(in_portions(r, "c", t, [n - 2, 2])[-1:], want, where, "two tokens")
        check(in_portions(r, "c", t, [n - 70, 70])[-1:], want, where, "a portion")


@pytest.mark.parametrize("where", WHERE)
def test_layers_read_the_keys_of_the_layer_that_is_named(tmp_path, where):
    """Three layers keep keys and values, two read those of the middle one: reading a neighbour's is another answer."""
    sizes = (4, 2, 24, 40, 16, 50, None)
    cfg = oracle.model([oracle.attn_layer(*sizes), oracle.attn_layer(*sizes), oracle.attn_layer(*sizes),
                        oracle.attn_layer(*sizes[:5], 70, None, kv_from=1), oracle.attn_layer(*sizes, kv_from=1)], width=48)
    w, t = oracle.random_weights(cfg, 3), tokens_of(cfg, 150, 5)
    want = oracle.logits(cfg, w, t)
    for j in (0, 2):
        other = json.loads(json.dumps(cfg))
        other["layers"][4]["mixer"]["kv_from"] = j
        assert error(oracle.logits(other, w, t).float(), want).mean() > 2 * LIMIT["bfloat16"]
    path = oracle.save(cfg, w, tmp_path)
    with Replay(path, where, blocks=10) as r:
        for portions in ([150], [2], [70, 1]):
            check(in_portions(r, "a", t, portions), want, where, str(portions))
        kept = r.core.executor.worker.runner.model.kept
        assert kept[3]["only"]["k"] is kept[1]["only"]["k"] and kept[4]["only"]["v"] is kept[1]["only"]["v"]
        assert len(r.core.executor.worker.runner.model.cache_tensors()) == 6


@pytest.mark.parametrize("where", WHERE)
def test_a_state_remembers(tmp_path, where):
    """Update gates nearly shut: what the first tokens left is still there hundreds of tokens later, however these came, and
    a slot that another request leaves behind is not."""
    cfg = oracle.model([oracle.gru_layer(40, None)], width=48)
    w = oracle.random_weights(cfg, 9)
    w["l0.mix.z.b"] = torch.full_like(w["l0.mix.z.b"], -11.0)
    z = 0.5 * w["l0.mix.z"].double()
    t = [x % 90 for x in tokens_of(cfg, 400, 4)]
    t[0] = 95
    # the gate of the first token opens wide
    h = oracle.layer_norm(w["embed"].double() * cfg["embedding"]["scale"], w["l0.norm1"].double(), w["l0.norm1.b"].double(),
                          cfg["norm"]["eps"])
    w["l0.mix.z"] = (z + torch.outer(torch.full((40,), 13.0).double(), h[95] / (h[95] @ h[95]))).to(torch.bfloat16)
    want = oracle.logits(cfg, w, t)
    lost = oracle.logits(cfg, w, t[1:])
    assert error(lost[-50:].float(), want[-50:]).median() > 2 * LIMIT["bfloat16"]
    path = oracle.save(cfg, w, tmp_path)
    with Replay(path, where, blocks=27, slots=1) as r:
        for portions in ([400], [1], [2, 17, 300, 1], [257, 143], [16], [15]):
            check(in_portions(r, "a", t, portions), want, where, str(portions))
        check(r.step([("b", t[1:], range(399))], ["b"]), lost, where, "a used slot")


# ---- generation through the public entry point -------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_greedy_generation(models, name, where):
    """Prompts longer than a step's budget, a pool small enough to preempt: the scheduler's own steps. fp32 gives the
    oracle's tokens; in bf16 every token's logit is close to the oracle's best one."""
    cfg, w, path = models(name, where)
    prompts = [tokens_of(cfg, n, 30 + n) for n in (70, 3, 1, 41, 20, 55)]
    llm = engine(path, where, num_gpu_blocks_override=14)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    kv = llm.llm_engine.core.kv
    assert kv.pool.num_free == 13 and kv.states.num_free == 4
    llm.shutdown()
    for p, o in zip(prompts, outs):
        got = list(o.outputs[0].token_ids)
        rows = oracle.logits(cfg, w, p + got)[len(p) - 1:-1]          # greedy: every token is the best behind those before it
        if where[1] == "float32":
            assert got == rows.argmax(-1).tolist()
        else:
            lost = rows.max(-1).values - rows[torch.arange(12), torch.as_tensor(got)]
            assert lost.max() < 4 * LIMIT["bfloat16"] * rows.pow(2).mean().sqrt()


@pytest.mark.parametrize("where", WHERE)
def test_sampling_and_log_probabilities(models, where):
    cfg, w, path = models("aligned", where)
    llm = engine(path, where)
    p = tokens_of(cfg, 60, 2)
    a, b = (llm.generate([p, p[:9]], SamplingParams(temperature=0.8, top_p=0.9, seed=7, max_tokens=6, ignore_eos=True))
            for _ in range(2))
    assert [x.outputs[0].token_ids for x in a] == [x.outputs[0].token_ids for x in b]
    out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=2, logprobs=3, prompt_logprobs=0, ignore_eos=True))[0]
    want = torch.log_softmax(oracle.logits(cfg, w, p), -1)
    tol = 1e-3 if where[1] == "float32" else 0.4
    for i in range(1, len(p)):
        assert abs(out.prompt_logprobs[i][p[i]] - want[i - 1, p[i]].item()) < tol
    first = out.outputs[0].logprobs[0]
    assert all(abs(v - want[-1, k].item()) < tol for k, v in first.items())
    llm.shutdown()


@gpu
@pytest.mark.parametrize("name", oracle.CONFIGS)
def test_cuda_graphs_replay_the_same_tokens(models, name):
    cfg, w, path = models(name, ("cuda", "bfloat16"))
    prompts = [tokens_of(cfg, n, 50 + n) for n in (40, 40, 7, 90)]
    sp = SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True)
    got = []
    for graphs in (False, True):
        llm = engine(path, ("cuda", "bfloat16"), tokenweave_cuda_graphs=graphs)
        got.append([o.outputs[0].token_ids for o in llm.generate(prompts, sp)])
        if graphs:
            assert llm.llm_engine.core.executor.worker.runner.graph_replays > 10
        llm.shutdown()
    assert got[0] == got[1]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("mode", [False, True])
def test_sleep_and_wake(models, where, mode):
    if mode and where[0] == "cpu":
        pytest.skip("released physical memory is the GPU's")
    cfg, w, path = models("aligned", where)
    llm = engine(path, where, enable_sleep_mode=mode)
    p, sp = tokens_of(cfg, 30, 1), SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True)
    before = llm.generate([p], sp)[0].outputs[0].token_ids
    llm.sleep(level=1)
    llm.wake_up()
    assert llm.generate([p], sp)[0].outputs[0].token_ids == before
    llm.shutdown()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("kw", [dict(enable_prefix_caching=True), dict(speculative_config=2)])
def test_cached_prefixes_and_drafts(models, where, kw):
    """A model whose layers keep no state takes over the blocks of a shared prompt and verifies drafts; others refuse."""
    cfg, w, path = models("attention", where)
    llm = engine(path, where, **kw)
    p = (tokens_of(cfg, 10, 4) * 5)[:50]
    for _ in range(2):
        out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))[0]
        if where[1] == "float32":
            assert list(out.outputs[0].token_ids) == oracle.greedy(cfg, w, p, 9)
    if "enable_prefix_caching" in kw:
        assert llm.llm_engine.core.kv.prefix_hits == 3
    llm.shutdown()
    with pytest.raises(ValueError, match="does not support"):
        EngineArgs(model=models("aligned", where)[2], **kw).create_engine_config()


# ---- configuration, loading, runner -----------------------------------------------------------------------------------
def changed(cfg, edit):
    cfg = json.loads(json.dumps(cfg))
    edit(cfg)
    return ModelConfig.from_hf_dict(cfg)


def test_config_reader(models):
    cfg, _, path = models("odd")
    m = ModelConfig.from_pretrained(path)
    assert m.architecture == "giforax" and m.block == "sandwich" and m.norm == "layer" and m.depth_average
    assert m.has_state and m.num_layers == 5 and m.embed_scale == 1.0 and m.rms_norm_eps == 1e-3 and not m.tie_word_embeddings
    assert not ModelConfig.from_pretrained(models("attention")[2]).has_state
    for edit in (lambda c: c["layers"][0].update(type="attention2"), lambda c: c["layers"][0]["mlp"].update(kind="sparse")):
        with pytest.raises(ValueError, match="unknown"):
            changed(cfg, edit)


@pytest.mark.parametrize("what,edit", [
    ("9 of 5 experts", lambda c: c["layers"][0]["mlp"]["router"].update(top=9)),
    ("an earlier layer", lambda c: c["layers"][3]["mixer"].update(kv_from=3)),
    ("an earlier layer", lambda c: c["layers"][3]["mixer"].update(kv_from=4)),
    ("an earlier layer", lambda c: c["layers"][3]["mixer"].update(kv_from=1)),       # a recurrence
    ("an earlier layer", lambda c: c["layers"][3]["mixer"].update(kv_from=0)),       # other sizes
    ("an earlier layer", lambda c: c["layers"][3]["mixer"]["rot"].update(base=31.0)),
    ("an earlier layer", lambda c: c["layers"].append({**c["layers"][3], "mixer": {**c["layers"][3]["mixer"], "kv_from": 3}})),
    ("rotated dimensions", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12))])
def test_models_that_do_not_exist(models, what, edit):
    with pytest.raises(ValueError, match=what):
        LLM(changed(models("odd")[0], edit), device="cpu", dtype="float32", skip_tokenizer_init=True)


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(quantization="fp8"), dict(enable_lora=True),
                                dict(pipeline_parallel_size=2)])
def test_refused_options(models, kw):
    with pytest.raises(ValueError, match="does not support"):
        EngineArgs(model=models("odd")[2], **kw).create_engine_config()


@pytest.mark.parametrize("fault", ["missing", "shape", "unknown", "shared"])
def test_loader_refuses_a_wrong_checkpoint(models, tmp_path, fault):
    cfg, w, _ = models("odd")
    w = dict(w)
    if fault == "missing":
        del w["l0.mix.pb"]
    elif fault == "shape":
        w["l1.dwa"] = w["l1.dwa"][:-1]
    elif fault == "shared":
        w["l3.mix.k"] = w["l2.mix.k"].clone()         # the layer reads another's keys
    else:
        w["l2.norm2"] = w["l0.norm1"].clone()         # the layer has no feed-forward
    with pytest.raises(ValueError):
        Replay(oracle.save(cfg, w, tmp_path), CPU, blocks=2)


def test_dummy_weights_and_reduced_layers():
    for n in (None, 3, 1):
        llm = LLM("tiny-giforax", device="cpu", dtype="float32", skip_tokenizer_init=True, max_num_batched_tokens=64,
                  max_model_len=128, num_hidden_layers_override=n)
        out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
        assert len(out[0].outputs[0].token_ids) == 4
        llm.shutdown()


def test_engine_core_process(models):
    cfg, w, path = models("aligned")
    llm = engine(path, CPU, engine_core_process=True)
    p = tokens_of(cfg, 30, 6)
    out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))[0]
    assert list(out.outputs[0].token_ids) == oracle.greedy(cfg, w, p, 4)
    llm.shutdown()


@pytest.mark.parametrize("where", WHERE)
def test_trace_runner_program(models, expected, tmp_path, where):
    cfg, w, path = models("odd", where)
    a, b = tokens_of(cfg, 70, 1), tokens_of(cfg, 5, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:2], "want": []}],
              "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": b, "want": [4]}, {"id": "a", "tokens": a[66:], "want": [3, 0]}],
              "end": ["a", "c"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", where[1], "--out",
                        str(tmp_path), "--max-tokens", "192", "--device", where[0]],
                       input="\n".join(map(json.dumps, steps)), capture_output=True, text=True, timeout=280)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    la, lb = expected("odd", where, a), expected("odd", where, b)
    for step, want in ((0, la[[0, 65]]), (2, torch.stack([lb[4], la[69], la[66]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(want.shape))
        check(got, want, where, f"step {step}")
    assert not (tmp_path / "1.f32").exists()


# ---- mechanisms alone ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims", [18, 16, 6])
@pytest.mark.parametrize("own", [True, False])
def test_rotation_and_unit_norm(dims, own):
    """Pairs of halves turn, whole heads but for the last dimensions, then every head is divided by its root mean square;
    a layer without keys of its own prepares queries only."""
    H, G, D, V, T, eps = 3, 1, 18, 8, 40, 1e-3
    rot = dict(base=200.0, dims=dims)
    part = GroupedAttention(dict(heads=H, kv_heads=G, dim=D, vdim=V, scale=1.0), eps, dtype=torch.float32, device="cpu", rot=rot,
                            qk_norm="unit", weights="sigmoid", chunk=7, head_gate=True, kv_from=None if own else 0)
    assert part.own_kv == (G if own else 0) and set(part.tensor_targets(4, None, None, None)) == {"q", "o", "pb", "g"} | (
        {"k", "v"} if own else set())
    from types import SimpleNamespace
    table = rope_table(SimpleNamespace(rope_tables={}, max_positions=64, device="cpu"), rot)
    m, nb = one_sequence(T)
    q, k, v = 0.1 * torch.randn(T, H, D), torch.randn(T, G, D), torch.randn(T, G, V)
    order = part.rot_order
    pad = lambda x: torch.nn.functional.pad(x[..., order], (0, 24 - D)).reshape(T, -1)
    kc, vc, got = torch.zeros(nb, 16, G, 24), torch.zeros(nb, 16, G, V), torch.zeros(T, H * 24)
    rows, caches = (torch.cat([pad(q), pad(k), v.view(T, -1)], 1), (kc, vc)) if own else (pad(q), (None, None))
    hops.qkv_prep(rows, H, part.own_kv, D, V, got, *caches, m, None, None, "unit", None, None, eps, 0.0, 1, table)
    at = m.slot_mapping.long()
    want = lambda x: oracle.unit(oracle.rotate(x.double(), rot), eps)[..., order]
    assert (got.view(T, H, 24)[..., :D] - want(q)).abs().max() < 1e-5
    if own:
        assert (kc.view(-1, G, 24)[at][..., :D] - want(k)).abs().max() < 1e-5 and torch.equal(vc.view(-1, G, V)[at], v)


@pytest.mark.parametrize("chunk", [1, 7, 16, 50, 100])
def test_sigmoid_weights_in_chunks(chunk):
    H, G, D, V, T, page = 6, 3, 16, 24, 50, 16
    m, nb = one_sequence(T, page)
    q, k, v = torch.randn(T, H, D), torch.randn(T, G, D), torch.randn(T, G, V)
    kc, vc, bias, gate = torch.zeros(nb, page, G, D), torch.zeros(nb, page, G, V), torch.randn(H) - 1, torch.randn(T, H + 2)
    kc.view(-1, G, D)[m.slot_mapping.long()], vc.view(-1, G, V)[m.slot_mapping.long()] = k, v
    out = torch.zeros(T, H * V)
    hops.grouped_attention(q.view(T, -1), kc, vc, out, m, H, G, 0.3, None, False, 1.0, key_bias=bias, chunk=chunk, gate=gate)
    want = oracle.sigmoid_attention(q.double(), k.double(), v.double(), 0.3, bias.double(), chunk)
    want = want * oracle.sigmoid(gate[:, :H].double())[:, :, None]
    assert (out - want.flatten(1)).abs().max() < 1e-5


def test_options_of_attention_that_do_not_go_together():
    sizes = dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0)
    for kw in (dict(chunk=4), dict(head_gate=True), dict(weights="sigmoid", window=3), dict(weights="sigmoid", sink=True),
               dict(weights="linear"), dict(qk_norm="other"), dict(kv_from=0, bias=True)):
        with pytest.raises(ValueError):
            GroupedAttention(sizes, 1e-5, dtype=torch.float32, device="cpu", **kw)


@pytest.mark.parametrize("portions", [[30], [1], [7, 2, 21]])
def test_min_gru(portions):
    from types import SimpleNamespace

    from tokenweave_b200.layers.mixers import MinGRUMixer
    W, I, T = 20, 13, 30
    mixer = MinGRUMixer(dict(width=I), W, 1e-5, dtype=torch.float32, device="cpu")
    w = {k: torch.randn(s) for k, (s, _) in mixer.tensor_targets().items()}
    for k, (_, put) in mixer.tensor_targets().items():
        put(w[k])
    h, kept, rows = torch.randn(T, 24), {}, []
    h[:, W:] = 0
    want, state = oracle.min_gru(h[:, :W].double(), {k: v.double() for k, v in w.items()})
    mixer.init_state(kept, 3)
    kept["state"].fill_(5.0)                          # what another sequence left
    rt = SimpleNamespace(buffer=lambda name, n, cols: torch.zeros(n, cols))
    at, i32, i = 0, lambda *x: torch.tensor(x, dtype=torch.int32), 0
    while at < T:
        n = min(portions[min(i, len(portions) - 1)], T - at)
        i += 1
        meta = SimpleNamespace(cu_q=i32(0, n), kv_lens=i32(at + n), extra={
            "state_slots": i32(1), "scan_seqs": i32(*([0] if n < 16 else [])), "chunk_seqs": i32(*([0] if n >= 16 else []))})
        out = torch.zeros(n, 24)
        mixer(h[at:at + n], meta, rt, out, kept)
        rows.append(out[:, :W])
        at += n
    assert (torch.cat(rows) - want).abs().max() < 1e-4 and (kept["state"][1, :I] - state).abs().max() < 1e-5
    assert (kept["state"][[0, 2]] == 5.0).all()


@pytest.mark.parametrize("kind", ["layer", "rms"])
def test_sandwich_norms_and_depth_average(kind):
    T, W, eps = 9, 21, 1e-3
    table, ids = torch.randn(11, 24) + 0.5, torch.randint(0, 11, (T,), dtype=torch.int32)
    norms = [(1 + 0.3 * torch.randn(W), torch.randn(W) if kind == "layer" else None) for _ in range(4)]

    def norm(x, wb):
        return (oracle.unit(x, eps) * wb[0] if kind == "rms"
                else oracle.layer_norm(x, wb[0].double(), wb[1].double(), eps))
    x, xa, results = torch.zeros(T, 24), torch.zeros(T, 24), torch.zeros(3, T, 24)
    hops.embed_sandwich(ids, table, 0.6, x, results[0], norms[0], eps, xa)
    want = [table[ids.long(), :W].double() * 0.6]
    stream = want[0]
    assert (xa[:, :W] - norm(stream, norms[0])).abs().max() < 1e-5
    for n in (1, 2, 3):
        y, coef = torch.randn(T, 24), torch.randn(n + 1)
        hops.sandwich_step(y, x, norms[1], norms[2], eps, xa)
        stream = stream + norm(y[:, :W].double(), norms[1])
        assert (xa[:, :W] - norm(stream, norms[2])).abs().max() < 1e-4
        hops.sandwich_step(y, x, norms[2], norms[3], eps, xa, coef, results, n == 3)
        want.append(stream + norm(y[:, :W].double(), norms[2]))
        stream = oracle.depth_average(coef.double(), want)
        assert (xa[:, :W] - norm(stream, norms[3])).abs().max() < 1e-4
    assert (x[:, :W] - stream).abs().max() < 1e-4 and (results[2, :, :W] - want[2]).abs().max() < 1e-4


@pytest.mark.parametrize("experts,top", [(6, 2), (6, 6), (40, 9), (1, 1)])
def test_router(experts, top):
    T, W = 30, 17
    h, w = torch.randn(T, W), torch.randn(experts, W)
    wts, ids, _ = reference.moe_route(h, w, experts, top, None, 0.0, "sigmoid", False)
    for t in range(T):
        want = dict(oracle.route(h[t].double(), w.double(), top))
        got = dict(zip(ids[t].tolist(), wts[t].tolist()))
        assert got.keys() == want.keys() and all(abs(got[e] - want[e]) < 1e-5 for e in want)


def test_the_weight_is_on_the_experts_input():
    T, W, ff, E, limit = 12, 16, 24, 5, 0.6
    h, gate, up, down = torch.randn(T, W), torch.randn(E, ff, W), torch.randn(E, ff, W), torch.randn(E, W, ff)
    wts, ids = torch.rand(T, 2), torch.stack([torch.randperm(E)[:2] for _ in range(T)]).int()
    res = {b: reference.moe_experts(h, torch.cat([gate, up], 1), down, wts, ids, ("clamped", limit, 1.702), b) for b in (True, False)}
    w = lambda e: {k: v[e].double() for k, v in (("gate", gate), ("up", up), ("down", down))}
    for t in range(T):
        x, pairs = h[t].double(), [(int(e), float(p)) for e, p in zip(ids[t], wts[t])]
        want = {True: sum(oracle.expert(p * x, w(e), limit) for e, p in pairs),
                False: sum(p * oracle.expert(x, w(e), limit) for e, p in pairs)}
        assert all((res[b][t] - want[b]).abs().max() < 1e-3 for b in want)
        assert (want[True] - want[False]).abs().max() > 0.1

"""Kebopel through the framework's engine (config reader, loader, cache and state manager, batch layout, kernels) against
the plain double-precision implementation of ``kebopel_oracle.py``. Every case runs on the CPU path in fp32 and, on a GPU,
in true fp32 and in bf16. The mechanisms alone are compared on the CPU here and kernel by kernel in
``test_grouped_ops_gpu.py``."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

import kebopel_oracle as oracle
from hybrid_testing import (LIMIT, WHERE, Replay, check, engine, error, gpu, in_portions, model_store, one_thread,
                            tokens_of, unequal_requests)
from tokenweave_b200 import LLM, SamplingParams
from tokenweave_b200.config import EngineArgs, ModelConfig
from tokenweave_b200.layers.attention import build_attention_metadata
from tokenweave_b200.models.hybrid import layer_runs
from tokenweave_b200.ops import hybrid as hops

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(autouse=True)
def _one_thread():
    yield from one_thread()


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return model_store(oracle, tmp_path_factory)


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", oracle.CONFIGS)
def test_whole_prompts(models, name, where):
    cfg, w, path = models(name)
    with Replay(path, where, blocks=20) as r:
        for n in (1, 2, 15, 64, 130, 290):
            t = tokens_of(cfg, n, n)
            check(r.step([("a", t, range(n))], ["a"]), oracle.logits(cfg, w, t), where, f"{n} tokens")


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", oracle.CONFIGS)
def test_portions_and_single_tokens(models, name, where):
    """However a prompt is cut - token by token, in twos, across pages, tiles and chunks - every position comes out alike."""
    cfg, w, path = models(name)
    t = tokens_of(cfg, 190, 3)
    want = oracle.logits(cfg, w, t)
    with Replay(path, where, blocks=13) as r:
        for portions in ([1], [2], [3, 2, 70, 2, 16, 17, 33], [64], [100, 1], [130, 2, 1]):
            check(in_portions(r, "a", t, portions), want, where, str(portions))


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_unequal_requests_share_steps_pages_and_slots(models, name, where):
    cfg, w, path = models(name)
    unequal_requests(oracle, cfg, w, path, where)


@pytest.mark.parametrize("where", WHERE)
def test_long_decoding(models, where):
    cfg, w, path = models("aligned")
    t = tokens_of(cfg, 420, 8)
    with Replay(path, where, blocks=28) as r:
        check(in_portions(r, "a", t, [20, 1]), oracle.logits(cfg, w, t), where)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("page", [16, 64, 128])
def test_page_sizes(models, where, page):
    cfg, w, path = models("odd")
    t = tokens_of(cfg, 250, 9)
    want = oracle.logits(cfg, w, t)
    with Replay(path, where, blocks=256 // page, page=page) as r:
        check(in_portions(r, "a", t, [page - 1, 2, page, 1, 1, 40]), want, where)


def test_the_residual_stream_after_every_layer_run(models, monkeypatch):
    """fp32 on the CPU: the stream behind every run of a layer, the passes of the loop one by one."""
    cfg, w, path = models("odd")
    t, got, want = tokens_of(cfg, 40, 2), [], []
    oracle.logits(cfg, w, t, want)
    plain = hops.add_prenorm_

    def spy(y, x32, first, weight, eps, xa):
        got.append(x32[:, :cfg["width"]] + y[:, :cfg["width"]])
        plain(y, x32, first, weight, eps, xa)
    monkeypatch.setattr(hops, "add_prenorm_", spy)
    with Replay(path, ("cpu", "float32"), blocks=4) as r:
        r.step([("a", t, [])], ["a"])
    assert len(got) == len(want) == len(layer_runs(4, cfg["loop"])) == 7
    for a, b in zip(got, want):
        assert (a - b.float()).abs().max() < 1e-4


# ---- keys far away ---------------------------------------------------------------------------------------------------------
def stand_out(cfg, weights, tokens, key, query):
    """Edits the first layer so that the score of (query, key) in its last head stands out: the query's projection gets a
    large component along the key. Norms take the component's size away, the configuration's scale gives it back."""
    layer, w = cfg["layers"][0], {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    pair = layer["type"] == "parallel"
    m, pre = (layer["mixer"]["left"], "l0.mix.left.") if pair else (layer["mixer"], "l0.mix.")
    h = oracle.rms_norm(oracle.embedding(tokens, w["embed"], w["bigram"], cfg["embedding"]["bigram"]), w["l0.norm1"], eps)
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k = h @ w[pre + "k"].T
    if pair:
        k = oracle.rms_norm(k, w[pre + "k.norm"], eps).view(len(tokens), G, D)[key, G - 1]
        along = k / w[pre + "q.norm"][-D:]
    else:
        k = oracle.short_conv(k + w[pre + "k.b"], w[pre + "k.conv"]).view(len(tokens), G, D)
        k = oracle.rms_norm(k, w[pre + "k.norm"], eps)[key, G - 1]
        along = k / w[pre + "q.norm"]
    q = w[pre + "q"].clone()
    q[-D:] += 300.0 / along.norm() * torch.outer(along, h[query] / (h[query] @ h[query]))
    o = w[pre + "o"].clone()
    o[:, -V:] *= 8                                    # the head carries the layer's output
    out = {**weights, pre + "q": q.to(torch.bfloat16), pre + "o": o.to(torch.bfloat16)}
    if not pair:                                      # the head's queries pass through the convolution as they are
        conv = w[pre + "q.conv"].clone()
        conv[-D:] = 0
        conv[-D:, -1] = 1
        out[pre + "q.conv"] = conv.to(torch.bfloat16)
    return out


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("kind", ["attention", "parallel"])
@pytest.mark.parametrize("key", [0, 1, 63, 64, 127, 128, 255, 256, 328])
def test_a_far_key_is_seen(tmp_path, where, kind, key):
    """The last position asks for one key far back - the first tokens, both sides of a page's and of a tile's edge - in
    a prompt and decoded alone. Without that key the answer would be another one."""
    layers = {"attention": oracle.attn_layer(4, 2, 24, 40, 56, every=100, scale=2.0),
              "parallel": oracle.parallel_layer((4, 2, 24, 40), (2, 16, 24), (0.9, 0.99), 56, scale=1.5)}
    cfg = oracle.model([layers[kind], oracle.parallel_layer((2, 1, 24, 16), (2, 24, 16), (0.5, 0.99), None)], width=48)
    n = 330 + 1
    t = [x % 90 for x in tokens_of(cfg, n, 21)]
    t[key], t[-1] = 95, 96                            # two tokens that occur once
    w = stand_out(cfg, oracle.random_weights(cfg, 4), t, key, n - 1)
    want = oracle.logits(cfg, w, t)[-1:]
    other = list(t)
    other[key] = 3
    assert error(oracle.logits(cfg, w, other)[-1:].float(), want)[0] > 2 * LIMIT["bfloat16"]
    path = oracle.save(cfg, w, tmp_path)
    with Replay(path, where, blocks=6, page=64) as r:
        check(r.step([("a", t, [n - 1])], ["a"]), want, where, "prompt")
        r.step([("b", t[:200], [])])
        r.step([("b", t[200:-1], [])])
        check(r.step([("b", t[-1:], [0])], ["b"]), want, where, "decoded")


@pytest.mark.parametrize("where", WHERE)
def test_a_state_remembers(tmp_path, where):
    """A lightning attention with hardly any decay: the first tokens still count hundreds of tokens later, in a prompt, in
    portions and decoded; and a slot that another sequence has used starts from nothing."""
    cfg = oracle.model([oracle.parallel_layer((1, 1, 8, 8), (3, 16, 24), (0.999, 1.0, 0.9995), None, (0.02, 1.0))], width=48)
    w = oracle.random_weights(cfg, 6)
    w["l0.mix.right.k"] = (w["l0.mix.right.k"].float() * 3).to(torch.bfloat16)
    t = tokens_of(cfg, 300, 11)
    for i in range(8, 300):
        t[i] = 5 + i % 2                              # nothing new after the first eight tokens
    want = oracle.logits(cfg, w, t)
    other = oracle.logits(cfg, w, [7] * 8 + t[8:])
    assert error(other[-1:].float(), want[-1:])[0] > 1e-3
    path = oracle.save(cfg, w, tmp_path)
    with Replay(path, where, blocks=20, slots=1) as r:
        for portions in ([300], [8, 292], [128, 1], [2, 5, 100, 16, 3]):
            check(in_portions(r, "a", t, portions), want, where, str(portions))


# ---- generation through the public entry point -------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_greedy_generation(models, name, where):
    """More requests than slots, prompts longer than a step's budget, a pool small enough to preempt: the scheduler's own
    steps. fp32 gives the oracle's tokens; in bf16 every token's logit is close to the oracle's best one."""
    cfg, w, path = models(name)
    prompts = [tokens_of(cfg, n, 30 + n) for n in (70, 3, 1, 41, 20, 55)]
    llm = engine(path, where, num_gpu_blocks_override=14)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    kv = llm.llm_engine.core.kv
    assert kv.states.num_free == 4 and kv.pool.num_free == 13
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
    cfg, w, path = models("aligned")
    llm = engine(path, where)
    p = tokens_of(cfg, 60, 2)
    a, b = (llm.generate([p, p[:9]], SamplingParams(temperature=0.8, top_p=0.9, seed=7, max_tokens=6, ignore_eos=True))
            for _ in range(2))
    assert [x.outputs[0].token_ids for x in a] == [x.outputs[0].token_ids for x in b]
    out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=2, logprobs=3, prompt_logprobs=0, ignore_eos=True))[0]
    want = torch.log_softmax(oracle.logits(cfg, w, p), -1)
    tol = 1e-3 if where[1] == "float32" else 0.25
    for i in range(1, len(p)):
        assert abs(out.prompt_logprobs[i][p[i]] - want[i - 1, p[i]].item()) < tol
    first = out.outputs[0].logprobs[0]
    assert all(abs(v - want[-1, k].item()) < tol for k, v in first.items())
    llm.shutdown()


@gpu
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_cuda_graphs_replay_the_same_tokens(models, name):
    cfg, w, path = models(name)
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
def test_sleep_and_wake(models, where):
    cfg, w, path = models("aligned")
    llm = engine(path, where)
    p, sp = tokens_of(cfg, 30, 1), SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True)
    before = llm.generate([p], sp)[0].outputs[0].token_ids
    llm.sleep(level=1)
    llm.wake_up()
    assert llm.generate([p], sp)[0].outputs[0].token_ids == before
    llm.shutdown()


# ---- configuration, loading, runner -----------------------------------------------------------------------------------
def test_config_reader(models):
    cfg, _, path = models("odd")
    m = ModelConfig.from_pretrained(path)
    assert m.architecture == "kebopel" and m.block == "parallel" and m.has_state and m.num_layers == 4
    assert m.loop == cfg["loop"] and m.bigram == cfg["embedding"]["bigram"]
    for change in ({"type": "attention2"}, {"mlp": {"kind": "sparse", "ff": 8}}):
        with pytest.raises(ValueError, match="unknown"):
            ModelConfig.from_hf_dict({**cfg, "layers": [{**cfg["layers"][0], **change}]})
    no_state = oracle.model([oracle.attn_layer(2, 1, 8, 8, None, conv=1)])
    assert not ModelConfig.from_hf_dict(no_state).has_state
    assert ModelConfig.from_hf_dict(oracle.CONFIGS["attention"]).has_state           # a convolution keeps inputs


def test_layer_runs():
    assert layer_runs(3, None) == [(0, False), (1, False), (2, False)]
    assert layer_runs(4, dict(start=1, stop=3, times=3)) == [(0, False), (1, False), (2, False), (1, True), (2, False),
                                                             (1, True), (2, False), (3, False)]
    assert layer_runs(2, dict(start=0, stop=2, times=1)) == [(0, False), (1, False)]
    for bad in (dict(start=1, stop=1, times=2), dict(start=0, stop=4, times=2), dict(start=0, stop=1, times=0)):
        with pytest.raises(ValueError, match="loop"):
            layer_runs(3, bad)


def test_every_pass_of_a_loop_has_its_own_cache_and_state(models):
    cfg, w, path = models("aligned")
    with Replay(path, ("cpu", "float32"), blocks=4) as r:
        model = r.core.executor.worker.runner.model
        n = len(layer_runs(3, cfg["loop"]))
        tensors = model.cache_tensors()
        assert len(model.kept) == n == 7 and len({t.data_ptr() for t in tensors}) == len(tensors)
        per_pass = sum(model.layers[i].mixer.cache_bytes_per_block(16) for i in (0, 1)) * 3
        assert model.kv_cache_bytes_per_block(16) == per_pass + model.layers[2].mixer.cache_bytes_per_block(16)
        held = sum(t.numel() * t.element_size() for t in tensors)
        assert held == model.kv_cache_bytes_per_block(16) * 5 + model.state_bytes_per_slot() * 4


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(enable_prefix_caching=True), dict(quantization="fp8"),
                                dict(speculative_config=2), dict(enable_lora=True), dict(pipeline_parallel_size=2)])
def test_refused_options(models, kw):
    with pytest.raises(ValueError, match="does not support"):
        EngineArgs(model=models("odd")[2], **kw).create_engine_config()


@pytest.mark.parametrize("kw", [dict(enable_prefix_caching=True), dict(speculative_config=2)])
def test_models_without_state_take_cached_prefixes_and_drafts(tmp_path, kw):
    """Attention only, no convolution state: blocks of a shared prompt are taken over (the token pair at its end comes from
    the prompt), and drafts are verified."""
    cfg = oracle.model([oracle.attn_layer(4, 2, 16, 24, 40, conv=1), oracle.attn_layer(2, 2, 8, 16, None, conv=1)],
                       loop=dict(start=0, stop=1, times=2))
    w = oracle.random_weights(cfg, 2)
    llm = engine(oracle.save(cfg, w, tmp_path), ("cpu", "float32"), **kw)
    p = (tokens_of(cfg, 10, 4) * 5)[:50]
    for _ in range(2):
        out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))[0]
        assert list(out.outputs[0].token_ids) == oracle.greedy(cfg, w, p, 9)
    if "enable_prefix_caching" in kw:
        assert llm.llm_engine.core.kv.prefix_hits == 3
    llm.shutdown()


@pytest.mark.parametrize("fault", ["missing", "shape", "unknown"])
def test_loader_refuses_a_wrong_checkpoint(models, tmp_path, fault):
    cfg, w, _ = models("odd")
    w = dict(w)
    if fault == "missing":
        del w["l1.mix.right.norm"]
    elif fault == "shape":
        w["l0.mix.k.conv"] = w["l0.mix.k.conv"][:-1]
    else:
        w["l0.norm2"] = w["l0.norm1"].clone()
    with pytest.raises(ValueError):
        Replay(oracle.save(cfg, w, tmp_path), ("cpu", "float32"), blocks=2)


def test_dummy_weights_and_reduced_layers():
    for n in (None, 2, 1):
        llm = LLM("tiny-kebopel", device="cpu", dtype="float32", skip_tokenizer_init=True, max_num_batched_tokens=64,
                  max_model_len=128, num_hidden_layers_override=n)
        out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
        assert len(out[0].outputs[0].token_ids) == 4
        llm.shutdown()


def test_engine_core_process(models):
    cfg, w, path = models("aligned")
    llm = engine(path, ("cpu", "float32"), engine_core_process=True)
    p = tokens_of(cfg, 30, 6)
    out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))[0]
    assert list(out.outputs[0].token_ids) == oracle.greedy(cfg, w, p, 4)
    llm.shutdown()


@pytest.mark.parametrize("where", WHERE)
def test_trace_runner_program(models, tmp_path, where):
    cfg, w, path = models("odd")
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
    la, lb = oracle.logits(cfg, w, a), oracle.logits(cfg, w, b)
    for step, want in ((0, la[[0, 65]]), (2, torch.stack([lb[4], la[69], la[66]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(want.shape))
        check(got, want, where, f"step {step}")
    assert not (tmp_path / "1.f32").exists()


# ---- mechanisms alone ------------------------------------------------------------------------------------------------------
def one_sequence(T, page=16):
    """Metadata of one sequence's whole prompt over pages in descending order."""
    n = (T + page - 1) // page
    table = np.arange(n, 0, -1)
    pos = np.arange(T)
    return build_attention_metadata([T], [T], pos, table[pos // page] * page + pos % page, table[None], torch.device("cpu"),
                                    plan=([], [], [], [], []), extra={"row_seq": pos * 0, "state_slots": [0],
                                                                      "prev_token": [-1]}), n + 1


def test_pair_rows():
    spec = dict(buckets=7, mul_prev=1000003, mul_cur=12)
    ids = torch.tensor([3, 96, 0, 96], dtype=torch.int32)
    m, _ = one_sequence(4)
    from tokenweave_b200.ops.reference_hybrid import pair_rows
    got = pair_rows(ids, m.extra["row_seq"], m.cu_q, m.extra["prev_token"], spec).tolist()
    assert got == [oracle.bigram_row(p, t, spec) for p, t in ((None, 3), (3, 96), (96, 0), (0, 96))] and got[0] == 7


@pytest.mark.parametrize("bias", [False, True])
@pytest.mark.parametrize("sink", [False, True])
def test_attention_options(bias, sink):
    H, G, D, V, T, page = 6, 3, 16, 24, 50, 16
    m, nb = one_sequence(T, page)
    q, k, v = torch.randn(T, H, D) * 2, torch.randn(T, G, D), torch.randn(T, G, V)
    kc, vc = torch.zeros(nb, page, G, D), torch.zeros(nb, page, G, V)
    kc.view(-1, G, D)[m.slot_mapping.long()], vc.view(-1, G, V)[m.slot_mapping.long()] = k, v
    slopes = torch.tensor([oracle.distance_slope(h, H) for h in range(H)]) if bias else None
    out = torch.zeros(T, H * V)
    hops.grouped_attention(q.view(T, -1), kc, vc, out, m, H, G, 0.3, slopes, sink, -1.5)
    want = oracle.causal_softmax(q.double(), k.double(), v.double(), 0.3, bias, sink) * -1.5
    assert (out - want).abs().max() < 1e-5


def test_convolution_norms_and_temperature():
    H, G, D, V, T, taps, page = 4, 2, 16, 8, 30, 3, 16
    m, nb = one_sequence(T, page)
    n = (H + G) * D + G * V
    p, w = torch.randn(T, n), torch.randn(taps, n)
    wq, wk = 1 + 0.3 * torch.randn(D), 1 + 0.3 * torch.randn(D)
    spec = dict(coef=0.7, every=4)
    kc, vc, q = torch.zeros(nb, page, G, D), torch.zeros(nb, page, G, V), torch.zeros(T, H * D)
    state = torch.full((1, taps - 1, n), 9.0)         # left behind by another sequence
    hops.qkv_prep(p, H, G, D, V, q, kc, vc, m, w, state, "head", wq, wk, 1e-3, spec["coef"], spec["every"])
    u = oracle.short_conv(p.double(), w.double().T)
    want_q = oracle.rms_norm(u[:, :H * D].view(T, H, D), wq.double(), 1e-3)
    want_q = want_q * torch.tensor([1 + 0.7 * math.log(math.floor((i + 1) / 4) + 1) for i in range(T)])[:, None, None]
    assert (q.view(T, H, D) - want_q).abs().max() < 1e-5
    at = m.slot_mapping.long()
    want_k = oracle.rms_norm(u[:, H * D:(H + G) * D].view(T, G, D), wk.double(), 1e-3)
    assert (kc.view(-1, G, D)[at] - want_k).abs().max() < 1e-5
    assert (vc.view(-1, G, V)[at] - u[:, (H + G) * D:].view(T, G, V)).abs().max() < 1e-5
    assert torch.equal(state[0], p[-2:])


def test_whole_norm():
    H, G, D, V, T = 3, 1, 8, 8, 12
    m, nb = one_sequence(T)
    p, wq, wk = torch.randn(T, (H + G) * D + G * V), torch.randn(H * D), torch.randn(G * D)
    kc, vc, q = torch.zeros(nb, 16, G, D), torch.zeros(nb, 16, G, V), torch.zeros(T, H * D)
    hops.qkv_prep(p, H, G, D, V, q, kc, vc, m, None, None, "whole", wq, wk, 1e-3, 0.0, 1)
    assert (q - oracle.rms_norm(p[:, :H * D], wq, 1e-3)).abs().max() < 1e-5
    got_k = kc.view(-1, G * D)[m.slot_mapping.long()]
    assert (got_k - oracle.rms_norm(p[:, H * D:(H + G) * D], wk, 1e-3)).abs().max() < 1e-5


def test_lightning_recurrence_norm_and_gate():
    H, N, V, T = 3, 8, 16, 25
    q, k, v, decay = torch.randn(T, H, N), torch.randn(T, H, N), torch.randn(T, H, V), torch.tensor([0.2, 0.9, 1.0])
    p = torch.cat([v.reshape(T, -1), k.reshape(T, -1), q.reshape(T, -1)], 1)
    state, y = torch.full((2, H, V, N), 5.0), torch.zeros(T, H * V)
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32)
    hops.decay_scan(p, decay, state, y, i32(0), i32(0, T), i32(T), i32(1))
    want = oracle.lightning(q.double(), k.double(), v.double(), decay.double())
    assert (y - want).abs().max() < 1e-4 and state[0].min() == 5.0
    g, w, out = torch.randn(T, H * V), torch.randn(H * V), torch.zeros(T, H * V)
    hops.norm_gate(y, g, w, H * V, 1e-5, 0.4, out)
    assert (out - 0.4 * oracle.rms_norm(want, w, 1e-5) * oracle.sigmoid(g)).abs().max() < 1e-5


def test_gated_product():
    x, w = torch.randn(9, 16), torch.randn(48, 16)
    out = torch.zeros(9, 24)
    hops.gated_product(x, w, "gelu_tanh", out, None)
    assert (out - oracle.gelu_tanh(x @ w[:24].T) * (x @ w[24:].T)).abs().max() < 1e-4

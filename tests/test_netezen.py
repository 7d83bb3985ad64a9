"""Netezen through the framework's engine (config reader, loader, cache manager, batch layout, kernels) against the plain
double-precision implementation of ``netezen_oracle.py``. Every case runs on the CPU path in fp32 and, on a GPU, in true
fp32 and in bf16. The mechanisms alone are compared on the CPU here and kernel by kernel in ``test_netezen_ops_gpu.py``."""
import json
import math
import os
import subprocess
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import netezen_oracle as oracle
from hybrid_testing import (LIMIT, WHERE, Replay, check, engine, error, gpu, in_portions, one_thread,
                            tokens_of, unequal_requests)
from tokenweave_b200 import LLM, SamplingParams
from tokenweave_b200.config import EngineArgs, ModelConfig
from tokenweave_b200.layers.attention import build_attention_metadata
from tokenweave_b200.layers.mixers import GroupedAttention, pair_order, rope_table
from tokenweave_b200.ops import hybrid as hops
from tokenweave_b200.ops import reference

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(autouse=True)
def _one_thread():
    yield from one_thread()


CPU = ("cpu", "float32")


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
    """However a prompt is cut - token by token, in twos, across pages, tiles and windows - every position comes out alike."""
    cfg, w, path = models(name, where)
    t = tokens_of(cfg, 190, 3)
    with Replay(path, where, blocks=13) as r:
        for portions in ([1], [2], [3, 2, 70, 2, 16, 17, 33], [64], [100, 1], [130, 2, 1]):
            check(in_portions(r, "a", t, portions), expected(name, where, t), where, str(portions))


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_unequal_requests_share_steps_and_pages(models, name, where):
    cfg, w, path = models(name, where)
    unequal_requests(oracle, cfg, w, path, where)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["aligned", "latent"])
def test_long_decoding(models, expected, name, where):
    """The windows pass over decoded tokens many times."""
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


@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_the_streams_after_every_layer(models, monkeypatch, name):
    """fp32 on the CPU: the sum of the streams behind every layer."""
    cfg, w, path = models(name)
    t, got, want = tokens_of(cfg, 40, 2), [], []
    oracle.logits(cfg, w, t, want)
    plain = hops.streams_step
    ends, at = set(), -1
    for layer in cfg["layers"]:
        at += 1 if layer["mlp"] is None else 2
        ends.add(at)
    calls = iter(range(at + 1))

    def spy(y, x, hc, mult, next_in, *rest):
        old = x.clone()
        plain(y, x, hc, mult, next_in, *rest)
        if next(calls) in ends:
            if next_in is None:                       # the last streams are not stored
                plain(y, old, hc, mult, torch.ones(cfg["streams"]), *rest)
                x = old
            got.append(x.sum(1)[:, :cfg["width"]].clone())
    monkeypatch.setattr(hops, "streams_step", spy)
    with Replay(path, ("cpu", "float32"), blocks=4) as r:
        r.step([("a", t, [])], ["a"])
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        assert (a - b.float()).abs().max() < 1e-4


# ---- windows, kept tokens, far keys ----------------------------------------------------------------------------------------
def stand_out(cfg, weights, tokens, key, query):
    """Edits the first layer so that the score of (query, key) in its last head stands out, rotated as they are: the query's
    projection gets a large component along the key."""
    w, m, eps = {k: v.double() for k, v in weights.items()}, cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    u = w["embed"][torch.as_tensor(tokens)] * w["l0.hc1.in"].sum()
    h = oracle.unit(u, eps) * (1 + w["l0.norm1"])
    back = lambda v: oracle.rotate(v.view(1, 1, -1), m["rot"], [key - query]).view(-1)
    H, D, V = m["heads"], m["dim"], m["vdim"]
    if cfg["layers"][0]["type"] == "attention":
        G, name, size = m["kv_heads"], "l0.mix.q", D
        along = back((h @ w["l0.mix.k"].T).view(len(tokens), G, D)[key, G - 1])
        reads = h[query]
    else:
        C, name, size = m["kv_rank"], "l0.mix.uq", D + m["rot_dim"]
        ckr = h[key] @ w["l0.mix.dkv"].T
        c = oracle.unit(ckr[:C], eps) * w["l0.mix.dkv.norm"]
        along = torch.cat([(c @ w["l0.mix.uk"].T).view(H, D)[-1], back(ckr[C:])])
        reads = oracle.unit(h[query] @ w["l0.mix.dq"].T, eps) * w["l0.mix.dq.norm"]
    q, o = w[name].clone(), w["l0.mix.o"].clone()
    q[-size:] += 40.0 / m["scale"] / (along @ along) * torch.outer(along, reads / (reads @ reads))
    o[:, -V:] *= 8                                    # the head carries the layer's output
    return {**weights, name: q.to(torch.bfloat16), "l0.mix.o": o.to(torch.bfloat16)}


def ask(tmp_path, where, layer, n, key, seen):
    """The last of n positions asks for one key - in a prompt, in portions and decoded. A key it sees decides the answer; one
    that it does not see would, were the mask one token off or absent."""
    cfg = oracle.model([layer], width=48, streams=3, mult=1.0)
    t = [x % 90 for x in tokens_of(cfg, n, 21)]
    t[key], t[-1] = 95, 96                            # two tokens that occur once
    w = stand_out(cfg, oracle.random_weights(cfg, 4), t, key, n - 1)
    want = oracle.logits(cfg, w, t)[-1:]
    wrong = json.loads(json.dumps(cfg))
    mask = wrong["layers"][0]["mixer"]["mask"]
    if seen and key < mask.get("keep_first", 0):
        mask["keep_first"] = key
    elif seen:
        mask["size"] = n - 1 - key
    else:
        mask["size"] = n - key
    assert error(oracle.logits(wrong, w, t)[-1:].float(), want)[0] > 2 * LIMIT["bfloat16"]
    path = oracle.save(cfg, w, tmp_path)
    with Replay(path, where, blocks=(n + 63) // 64, page=64) as r:
        check(r.step([("a", t, [n - 1])], ["a"]), want, where, "prompt")
        r.step([("b", t[:n // 2], [])])
        r.step([("b", t[n // 2:-1], [])])
        check(r.step([("b", t[-1:], [0])], ["b"]), want, where, "decoded")
        check(in_portions(r, "c", t, [n - 2, 2])[-1:], want, where, "two tokens")
        check(in_portions(r, "c", t, [n - 70, 70])[-1:], want, where, "a portion")


LAST = 330                                            # the asking position


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("window,keep,key,seen", [
    (60, 0, LAST - 59, True), (60, 0, LAST - 60, False), (129, 0, LAST - 128, True), (129, 0, LAST - 129, False),
    (128, 4, LAST - 127, True), (128, 4, LAST - 128, False), (75, 4, 0, True), (75, 4, 3, True), (75, 4, 4, False),
    (75, 130, 127, True), (75, 130, 129, True), (75, 130, 130, False), (331, 0, 0, True), (330, 0, 0, False), (330, 1, 0, True),
    (203, 2, 128, True), (203, 2, 127, False), (267, 0, 64, True), (267, 0, 63, False), (1, 3, 2, True), (1, 3, 3, False),
    (2, 0, LAST - 1, True)])
def test_attention_sees_its_window_and_the_first_tokens(tmp_path, where, window, keep, key, seen):
    ask(tmp_path, where, oracle.attn_layer(4, 2, 24, 40, 16, window, keep, None), LAST + 1, key, seen)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("window,key,seen", [
    (40, LAST - 39, True), (40, LAST - 40, False), (129, LAST - 128, True), (129, LAST - 129, False), (331, 0, True),
    (330, 0, False), (203, 128, True), (203, 127, False), (267, 64, True), (267, 63, False), (2, LAST - 1, True)])
def test_latent_attention_sees_its_window(tmp_path, where, window, key, seen):
    ask(tmp_path, where, oracle.latent_layer(3, 24, 16, 16, 40, 32, window, None), LAST + 1, key, seen)


@pytest.mark.parametrize("where", WHERE)
def test_the_sink_counts_once(tmp_path, where):
    """Few visible keys and sinks above, near and below their scores: the answer without the sinks is another one."""
    cfg = oracle.model([oracle.latent_layer(4, 16, 8, 24, 32, 24, 3, None)], width=48, streams=2, mult=1.0)
    w = oracle.random_weights(cfg, 6)
    w["l0.mix.sink"] = torch.tensor([9.0, 1.0, -2.0, 30.0]).to(torch.bfloat16)
    t = tokens_of(cfg, 150, 11)
    want = oracle.logits(cfg, w, t)
    none = oracle.logits(cfg, {**w, "l0.mix.sink": torch.full((4,), -100.0)}, t)
    assert error(none.float(), want).min() > 2 * LIMIT["bfloat16"]
    path = oracle.save(cfg, w, tmp_path)
    with Replay(path, where, blocks=10) as r:
        for portions in ([150], [2], [70, 1]):
            check(in_portions(r, "a", t, portions), want, where, str(portions))


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
    assert llm.llm_engine.core.kv.pool.num_free == 13
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
    # in bf16 relative to the logits, which the tied embedding makes large
    tol = 1e-3 if where[1] == "float32" else 0.1 * oracle.logits(cfg, w, p).abs().max().item()
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
def test_sleep_and_wake(models, where):
    cfg, w, path = models("aligned", where)
    llm = engine(path, where)
    p, sp = tokens_of(cfg, 30, 1), SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True)
    before = llm.generate([p], sp)[0].outputs[0].token_ids
    llm.sleep(level=1)
    llm.wake_up()
    assert llm.generate([p], sp)[0].outputs[0].token_ids == before
    llm.shutdown()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("kw", [dict(enable_prefix_caching=True), dict(speculative_config=2)])
def test_cached_prefixes_and_drafts(models, where, kw):
    """No layer keeps a state: blocks of a shared prompt are taken over, and drafts are verified."""
    cfg, w, path = models("aligned", where)
    llm = engine(path, where, **kw)
    p = (tokens_of(cfg, 10, 4) * 5)[:50]
    for _ in range(2):
        out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))[0]
        if where[1] == "float32":
            assert list(out.outputs[0].token_ids) == oracle.greedy(cfg, w, p, 9)
    if "enable_prefix_caching" in kw:
        assert llm.llm_engine.core.kv.prefix_hits == 3
    llm.shutdown()


# ---- configuration, loading, runner -----------------------------------------------------------------------------------
def test_config_reader(models):
    cfg, _, path = models("odd")
    m = ModelConfig.from_pretrained(path)
    assert m.architecture == "netezen" and m.block == "streams" and not m.has_state and m.num_layers == 4
    assert m.streams == 3 and m.residual_mult == 1.0 and m.norm_offset == 1.0 and m.tie_word_embeddings
    for change in ({"type": "attention2"}, {"mlp": {"kind": "sparse", "ff": 8}}):
        with pytest.raises(ValueError, match="unknown"):
            ModelConfig.from_hf_dict({**cfg, "layers": [{**cfg["layers"][0], **change}]})
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["router"]["top"] = 9
    with pytest.raises(ValueError, match="9 of 5 experts"):
        EngineArgs(model=ModelConfig.from_hf_dict(bad), device="cpu").create_engine_config() and LLM(
            ModelConfig.from_hf_dict(bad), device="cpu", dtype="float32", skip_tokenizer_init=True)


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(quantization="fp8"), dict(enable_lora=True),
                                dict(pipeline_parallel_size=2)])
def test_refused_options(models, kw):
    with pytest.raises(ValueError, match="does not support"):
        EngineArgs(model=models("odd")[2], **kw).create_engine_config()


@pytest.mark.parametrize("fault", ["missing", "shape", "unknown"])
def test_loader_refuses_a_wrong_checkpoint(models, tmp_path, fault):
    cfg, w, _ = models("odd")
    w = dict(w)
    if fault == "missing":
        del w["l0.mix.sink"]
    elif fault == "shape":
        w["l0.hc2.mix"] = w["l0.hc2.mix"][:-1]
    else:
        w["l2.norm2"] = w["l0.norm1"].clone()         # the layer has no feed-forward
    with pytest.raises(ValueError):
        Replay(oracle.save(cfg, w, tmp_path), ("cpu", "float32"), blocks=2)


def test_dummy_weights_and_reduced_layers():
    for n in (None, 2, 1):
        llm = LLM("tiny-netezen", device="cpu", dtype="float32", skip_tokenizer_init=True, max_num_batched_tokens=64,
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
def one_sequence(T, page=16):
    """Metadata of one sequence's whole prompt over pages in descending order."""
    n = (T + page - 1) // page
    table = np.arange(n, 0, -1)
    pos = np.arange(T)
    return build_attention_metadata([T], [T], pos, table[pos // page] * page + pos % page, table[None], torch.device("cpu"),
                                    plan=([], [], [], [], []), extra={"row_seq": pos * 0}), n + 1


@pytest.mark.parametrize("scaling", [None, dict(factor=4.0, original=64, fast=16.0, slow=1.0),
                                     dict(factor=8.0, original=300, fast=2.0, slow=2.0),
                                     dict(factor=2.0, original=10 ** 5, fast=32.0, slow=0.1)])
@pytest.mark.parametrize("dims", [16, 6])
def test_rotation(dims, scaling):
    """Whole heads but for the last two dimensions, neighbouring pairs; queries and keys alike, values untouched."""
    H, G, D, V, T = 3, 1, 18, 8, 40
    rot = dict(base=200.0, dims=dims, scaling=scaling)
    table = rope_table(SimpleNamespace(rope_tables={}, max_positions=64, device="cpu"), rot)
    m, nb = one_sequence(T)
    q, k, v = torch.randn(T, H, D), torch.randn(T, G, D), torch.randn(T, G, V)
    pad = lambda x: torch.nn.functional.pad(x, (0, 24 - D)).reshape(T, -1)
    kc, vc, got = torch.zeros(nb, 16, G, 24), torch.zeros(nb, 16, G, V), torch.zeros(T, H * 24)
    hops.qkv_prep(torch.cat([pad(q), pad(k), v.view(T, -1)], 1), H, G, D, V, got, kc, vc, m, None, None, None, None, None, 1e-3,
                  0.0, 1, table)
    at = m.slot_mapping.long()
    assert (got.view(T, H, 24)[..., :D] - oracle.rotate(q.double(), rot)).abs().max() < 1e-5
    assert (kc.view(-1, G, 24)[at][..., :D] - oracle.rotate(k.double(), rot)).abs().max() < 1e-5
    assert torch.equal(vc.view(-1, G, V)[at], v)


def test_pairs_of_halves_are_the_same_rotation_in_another_order():
    order = pair_order(6, 9, True)
    assert order.tolist() == [0, 2, 4, 1, 3, 5, 6, 7, 8] and pair_order(6, 9, False)[order].tolist() == list(range(9))
    rot = dict(base=50.0, dims=6)
    x = torch.randn(5, 2, 9).double()
    turned = oracle.rotate(x, rot)
    f, _ = oracle.frequencies(rot)
    h = x[..., order]
    for p in range(5):
        for i in range(3):
            c, s = math.cos(p * f[i]), math.sin(p * f[i])
            assert torch.allclose(turned[p, :, order][:, i], h[p, :, i] * c - h[p, :, i + 3] * s)
            assert torch.allclose(turned[p, :, order][:, i + 3], h[p, :, i + 3] * c + h[p, :, i] * s)
    # a layer whose design turns halves: its weights are stored so that the kernel's neighbouring pairs are the design's
    sizes = dict(heads=2, kv_heads=1, dim=9, vdim=8, scale=1.0)
    kw = dict(dtype=torch.float32, device="cpu", rot=rot, bias=True, qk_norm="head")
    rows = {}
    for neighbours in (True, False):
        part = GroupedAttention(sizes, 1e-5, neighbour_pairs=neighbours, **kw)
        put = part.tensor_targets(4, lambda t, row: rows.setdefault((neighbours, row), t.clone()), lambda t, row: None, None)
        put["q"][1](torch.arange(18.0)[:, None].expand(18, 4))
        put["q.norm"][1](torch.arange(9.0))
        rows[neighbours] = part.q_norm_w[:9].tolist()
    back = pair_order(6, 9, False).tolist()
    assert rows[(True, 0)][:, 0].tolist() == list(range(9)) and rows[(False, 0)][:, 0].tolist() == back == rows[False]
    assert rows[(False, 16)][:, 0].tolist() == [9 + i for i in back]


@pytest.mark.parametrize("window,keep", [(1, 0), (7, 0), (16, 3), (50, 0), (20, 33), (100, 5)])
def test_window_with_kept_first_keys(window, keep):
    H, G, D, V, T, page = 6, 3, 16, 24, 50, 16
    m, nb = one_sequence(T, page)
    q, k, v = torch.randn(T, H, D) * 2, torch.randn(T, G, D), torch.randn(T, G, V)
    kc, vc = torch.zeros(nb, page, G, D), torch.zeros(nb, page, G, V)
    kc.view(-1, G, D)[m.slot_mapping.long()], vc.view(-1, G, V)[m.slot_mapping.long()] = k, v
    out = torch.zeros(T, H * V)
    hops.grouped_attention(q.view(T, -1), kc, vc, out, m, H, G, 0.3, None, False, 1.0, window=window, keep=keep)
    want = oracle.masked_softmax(q.double(), k.double(), v.double(), 0.3, window, keep)
    assert (out - want).abs().max() < 1e-5


@pytest.mark.parametrize("window", [1, 6, 40])
def test_latent_window_and_sink(window):
    """The absorbed form: every head's query for a cache row, the row's latent as the value."""
    H, C, R, T, page = 3, 16, 8, 30, 16
    m, nb = one_sequence(T, page)
    rows, qa, sink = torch.randn(T, C + R), torch.randn(T, H, C + R), torch.tensor([2.0, -1.0, 12.0])
    cache = torch.zeros(nb, page, C + R)
    cache.view(-1, C + R)[m.slot_mapping.long()] = rows
    out = torch.zeros(T, H, C)
    idx = torch.arange(T, dtype=torch.int32)
    hops.latent_attention(qa, cache, idx * 0, idx + 1, T, m.block_table, C, 0.4, out, T, window=window, sink=sink)
    want = oracle.masked_softmax(qa.double(), rows[:, None].double(), rows[:, None, :C].double(), 0.4, window, sink=sink)
    assert (out.view(T, -1) - want).abs().max() < 1e-5


@pytest.mark.parametrize("streams", [1, 3, 6])
def test_hyper_connections(streams):
    T, W, eps = 9, 21, 1e-3
    table, ids, y = torch.randn(11, 24), torch.randint(0, 11, (T,), dtype=torch.int32), torch.randn(T, 24)
    hc = {"in": torch.randn(streams), "out": torch.randn(streams), "mix": torch.randn(streams, streams)}
    nxt, w = torch.randn(streams), 0.3 * torch.randn(W)
    x, xa = torch.zeros(T, streams, 24), torch.zeros(T, 24)
    hops.embed_streams(ids, table, x, hc["in"], w, 1.0, eps, xa)
    old = torch.stack([table[ids.long(), :W].double()] * streams)
    seen = []
    wide = {k: v.double() for k, v in hc.items()}
    new = oracle.connect(old, wide, lambda u: (seen.append(oracle.unit(u, eps) * (1 + w)), y[:, :W].double())[1], 0.7)
    assert (xa[:, :W] - seen[0]).abs().max() < 1e-5
    last = x.clone()
    hops.streams_step(y, last, hc, 0.7, None, w, 1.0, eps, xa, first=True)
    assert (xa[:, :W] - oracle.unit(new.sum(0), eps) * (1 + w)).abs().max() < 1e-4
    hops.streams_step(y, x, hc, 0.7, nxt, w, 1.0, eps, xa, first=True)
    assert (x.transpose(0, 1)[..., :W] - new).abs().max() < 1e-5
    u = sum(nxt[s].double() * new[s] for s in range(streams))
    assert (xa[:, :W] - oracle.unit(u, eps) * (1 + w)).abs().max() < 1e-4
    # and once more, from streams that differ
    again = oracle.connect(new, wide, lambda _: y[:, :W].double(), 0.7)
    hops.streams_step(y, x, hc, 0.7, nxt, w, 1.0, eps, xa)
    assert (x.transpose(0, 1)[..., :W] - again).abs().max() < 1e-4


@pytest.mark.parametrize("experts,top", [(6, 2), (6, 6), (40, 9), (1, 1)])
def test_router(experts, top):
    T, W = 30, 17
    h, w = torch.randn(T, W), {"router": torch.randn(experts, W), "correction": 0.5 * torch.rand(experts)}
    sg = torch.randn(1, W)
    wts, ids, gate = reference.moe_route(h, torch.cat([w["router"], sg]), experts, top, w["correction"], 1e-20)
    changed = 0
    for t in range(T):
        want = dict(oracle.route(h[t].double(), {k: v.double() for k, v in w.items()}, top))
        got = dict(zip(ids[t].tolist(), wts[t].tolist()))
        assert got.keys() == want.keys() and all(abs(got[e] - want[e]) < 1e-5 for e in want)
        plain = (w["router"] @ h[t]).topk(top).indices.tolist()
        changed += set(plain) != set(got)
    assert changed > 0 or top == experts                 # the correction decides some choices
    assert (gate[:, 0] - oracle.sigmoid(h @ sg[0])).abs().max() < 1e-5


def test_feed_forwards():
    T, W, ff, limit = 12, 16, 24, 0.6
    h, up, gate, down = torch.randn(T, W), torch.randn(ff, W), torch.randn(ff, W), torch.randn(W, ff)
    a = torch.zeros(T, ff)
    hops.projection(h, up, None, (0, ff), a, "relu2")
    assert (a @ down.T - oracle.squared_relu_ff(h.double(), {"up": up.double(), "down": down.double()})).abs().max() < 1e-3
    hops.gated_product(h, torch.cat([gate, up]), ("clamped", limit, 1.702), a, None)
    want = oracle.clamped_ff(h.double(), {k: v.double() for k, v in (("gate", gate), ("up", up), ("down", down))}, limit)
    assert (a @ down.T - want).abs().max() < 1e-3

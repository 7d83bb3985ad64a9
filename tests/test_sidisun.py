"""Sidisun through the framework's engine (config reader, loader, cache and state manager, batch layout, kernels) against
the plain double-precision implementation of ``sidisun_oracle.py``. Every case runs on the CPU path in fp32 and, on a
GPU, in true fp32 and in bf16."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import sidisun_oracle as oracle
from hybrid_testing import (LIMIT, WHERE, Replay, check, engine, error, gpu, in_portions, model_store, one_thread,
                            tokens_of, unequal_requests)
from tokenweave_b200 import LLM, SamplingParams
from tokenweave_b200.config import EngineArgs, ModelConfig

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(autouse=True)
def _one_thread():
    yield from one_thread()


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return model_store(oracle, tmp_path_factory)


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


def stand_out(cfg, weights, tokens, key, query, gain):
    """Edits the first layer (latent attention on the embeddings) so that in head 0 the score of (query, key) grows by
    ``gain``: a rank-one change of the query map along the key's unrotated part."""
    m, w = cfg["layers"][0]["mixer"], {k: v.double() for k, v in weights.items()}
    e = w["embed"][torch.as_tensor(tokens)]
    c = oracle.rms_unit(e[key] @ w["l0.mix.dkv"][:m["kv_rank"]].T, cfg["norm"]["eps"]) * w["l0.mix.dkv.norm"]
    k = (c @ w["l0.mix.uk"].T)[:m["dim"]]
    q = oracle.rms_unit(e[query] @ w["l0.mix.dq"].T, cfg["norm"]["eps"]) * w["l0.mix.dq.norm"]
    uq = w["l0.mix.uq"].clone()
    uq[:m["dim"]] += gain / (m["scale"] * (k @ k)) * torch.outer(k, q / (q @ q))
    o = w["l0.mix.o"].clone()
    o[:, :m["vdim"]] *= 8                             # the head carries the layer's output
    return {**weights, "l0.mix.uq": uq.to(torch.bfloat16), "l0.mix.o": o.to(torch.bfloat16)}


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("key", [0, 1, 63, 64, 255, 256, 329])
def test_a_far_key_is_seen(tmp_path, where, key):
    """The last position asks for one key far back - the first tokens, both sides of a page's and of a tile's edge - in
    a prompt and decoded alone. Without that key the answer would be another one."""
    cfg = oracle.model([oracle.attn_layer(3, 24, 16, 24, 40, 32, 56, scaling=oracle.YARN),
                        oracle.mamba_layer(2, 24, 16, 1, None)], width=48)
    n = 330 + 1
    t = tokens_of(cfg, n, 21)
    t = [x % 90 for x in t]
    t[key], t[-1] = 95, 96                            # two tokens that occur once
    w = stand_out(cfg, oracle.random_weights(cfg, 4), t, key, n - 1, 60.0)
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


# ---- generation through the public entry point ----------------------------------------------------------------------


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
        if where[1] == "float32":
            assert got == oracle.greedy(cfg, w, p, 12)
        else:
            rows = oracle.logits(cfg, w, p + got)[len(p) - 1:-1]
            lost = rows.max(-1).values - rows[torch.arange(12), torch.as_tensor(got)]
            assert lost.max() < 4 * LIMIT["bfloat16"] * rows.pow(2).mean().sqrt()


@pytest.mark.parametrize("where", WHERE)
def test_sampling_log_probabilities_and_pooling(models, where):
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


# ---- configuration, loading, runner ----------------------------------------------------------------------------------
def test_config_reader(models):
    cfg, _, path = models("odd")
    m = ModelConfig.from_pretrained(path)
    assert m.architecture == "sidisun" and m.has_state and m.num_layers == 4 and m.logit_scale == cfg["logit_scale"]
    assert not ModelConfig.from_hf_dict(oracle.CONFIGS["attention"]).has_state
    with pytest.raises(ValueError, match="unsupported architecture"):
        ModelConfig.from_hf_dict({"architecture": "Nobody"})


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(enable_prefix_caching=True), dict(quantization="fp8"),
                                dict(speculative_config=2), dict(enable_lora=True), dict(pipeline_parallel_size=2)])
def test_refused_options(models, kw):
    with pytest.raises(ValueError, match="does not support"):
        EngineArgs(model=models("odd")[2], **kw).create_engine_config()


def test_prefix_caching_without_recurrent_layers(models):
    """A model of attention layers only keeps no state: cached blocks of a shared prompt are taken over."""
    cfg, w, path = models("attention")
    llm = engine(path, ("cpu", "float32"), enable_prefix_caching=True)
    p = tokens_of(cfg, 50, 4)
    for _ in range(2):
        out = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))[0]
        assert list(out.outputs[0].token_ids) == oracle.greedy(cfg, w, p, 5)
    assert llm.llm_engine.core.kv.prefix_hits == 3
    llm.shutdown()


@pytest.mark.parametrize("fault", ["missing", "shape", "unknown"])
def test_loader_refuses_a_wrong_checkpoint(models, tmp_path, fault):
    cfg, w, _ = models("odd")
    w = dict(w)
    if fault == "missing":
        del w["l1.mix.D"]
    elif fault == "shape":
        w["l0.mix.uk"] = w["l0.mix.uk"][:-1]
    else:
        w["l0.mix.extra"] = w["l0.norm1"].clone()
    with pytest.raises(ValueError):
        Replay(oracle.save(cfg, w, tmp_path), ("cpu", "float32"), blocks=2)


def test_dummy_weights_and_reduced_layers():
    for n in (None, 2):
        llm = LLM("tiny-sidisun", device="cpu", dtype="float32", skip_tokenizer_init=True, max_num_batched_tokens=64,
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
    cfg, w, path = models("aligned")
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

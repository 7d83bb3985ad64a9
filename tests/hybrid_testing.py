"""What the engine tests of the hybrid designs share: models made once per module, a replayer over a small pool, and the
comparison of logits with an oracle's."""
import numpy as np
import pytest
import torch

from tokenweave_b200 import LLM
from tokenweave_b200.config import EngineArgs
from tokenweave_b200.engine.core import EngineCore
from tokenweave_b200.engine.replay import StepReplayer

gpu = pytest.mark.gpu
WHERE = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="fp32", marks=gpu),
         pytest.param(("cuda", "bfloat16"), id="bf16", marks=gpu)]
# rms error of a position's logits over the rms of the logits. bf16: a softmax between two nearly equal keys can turn on
# one rounding, so single positions of a long prompt may be further off
LIMIT = {"float32": 1e-4, "bfloat16": 0.12}
TYPICAL, OUTLIER = 0.06, 0.3


def one_thread():
    """The oracles' products are tiny: several threads only get in each other's way. (Body of an autouse fixture.)"""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def model_store(oracle, tmp_path_factory):
    """name -> (config, weights, folder), each made once."""
    made = {}

    def get(name):
        if name not in made:
            cfg = oracle.CONFIGS[name]
            w = oracle.random_weights(cfg, seed=len(name))
            made[name] = (cfg, w, oracle.save(cfg, w, tmp_path_factory.mktemp(name)))
        return made[name]
    return get


def tokens_of(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class Replay:
    """A replayer over a small pool: ``blocks`` pages of ``page`` tokens, ``slots`` requests at a time."""

    def __init__(self, path, where, blocks, page=16, slots=4):
        device, dtype = where
        self.core = EngineCore(EngineArgs(
            model=path, dtype=dtype, device=device, skip_tokenizer_init=True, block_size=page, max_num_seqs=slots,
            num_gpu_blocks_override=blocks + 1, max_model_len=blocks * page,
            max_num_batched_tokens=blocks * page).create_engine_config())
        self.replayer = StepReplayer(self.core)

    def __enter__(self):
        return self.replayer

    def __exit__(self, *_):
        self.core.shutdown()


def error(got, want):
    want = want.float()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt())


def check(got, want, where, what=""):
    e = error(got, want)
    lim = LIMIT[where[1]]
    if where[1] == "bfloat16" and len(e) > 10:
        assert (e > TYPICAL).sum() <= max(1, 0.02 * len(e)), f"{what}: positions {(e > TYPICAL).nonzero().flatten().tolist()}"
        lim = OUTLIER
    assert e.max() < lim, f"{what}: position {int(e.argmax())} is off by {e.max():.2e} (limit {lim})"


def in_portions(replayer, rid, tokens, portions):
    """Feeds the tokens in portions of the given sizes (the last one repeats); logits of every position."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        part = tokens[at:at + portions[min(i, len(portions) - 1)]]
        at, i = at + len(part), i + 1
        out.append(replayer.step([(rid, part, range(len(part)))], [rid] if at == len(tokens) else []))
    return torch.cat(out)


def unequal_requests(oracle, cfg, w, path, where):
    """Up to three live requests in a pool that only fits by reusing what finished requests gave back; portions beside
    single tokens, requests left out of some steps. Every position is compared with the request alone."""
    rng = np.random.default_rng(5)
    lengths = [150, 9, 40, 2, 97, 64, 33, 1]
    todo = [(f"r{i}", tokens_of(cfg, n, 10 + i)) for i, n in enumerate(lengths)]
    got = {rid: [] for rid, _ in todo}
    live, at, waiting = {}, {}, list(todo)
    with Replay(path, where, blocks=19, slots=3) as r:
        while live or waiting:
            while waiting and len(live) < 3:
                rid, t = waiting[0]
                held = sum((len(x) + 15) // 16 for x in live.values())
                if held + (len(t) + 15) // 16 > 19:
                    break
                live[rid], at[rid] = t, 0
                waiting.pop(0)
            entries, end = [], []
            for rid, t in live.items():
                if len(live) > 1 and rng.random() < 0.2:
                    continue
                n = min(int(rng.choice([1, 1, 2, 3, 16, 30, 70])), len(t) - at[rid])
                entries.append((rid, t[at[rid]:at[rid] + n], range(n)))
                at[rid] += n
                if at[rid] == len(t):
                    end.append(rid)
            if not entries:
                continue
            logits = r.step(entries, end)
            for rid, part, _ in entries:
                got[rid].append(logits[:len(part)])
                logits = logits[len(part):]
            for rid in end:
                del live[rid]
        states = r.core.kv.states                      # None in models without recurrent state
        assert (states is None or states.num_free == 3) and r.core.kv.pool.num_free == 19
    for rid, t in todo:
        check(torch.cat(got[rid]), oracle.logits(cfg, w, t), where, rid)


def engine(path, where, **kw):
    device, dtype = where
    kw = {"block_size": 16, "num_gpu_blocks_override": 40, "max_model_len": 256, "max_num_batched_tokens": 48,
          "max_num_seqs": 4, **kw}
    return LLM(path, device=device, dtype=dtype, skip_tokenizer_init=True, **kw)

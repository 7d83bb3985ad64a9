"""The hybrid operators' plain PyTorch forms (the CPU path, and the reference of the kernel tests) against the mechanisms
of the independent oracle, one by one, plus the state-slot pool and the routing of a step's rows."""
import numpy as np
import pytest
import torch

import sidisun_oracle as oracle
from tokenweave_b200.config import EngineArgs
from tokenweave_b200.engine.kv_cache import KVCacheManager, StateSlotPool
from tokenweave_b200.engine.request import Request
from tokenweave_b200.ops import hybrid as hops
from tokenweave_b200.ops import reference
from tokenweave_b200.sampling_params import SamplingParams

EPS = 1e-4


def close(a, b, tol=2e-5):
    torch.testing.assert_close(a.double(), b.double(), atol=tol, rtol=tol)


def i32(x):
    return torch.as_tensor(x, dtype=torch.int32)


@pytest.mark.parametrize("scaling", [None, dict(factor=4.0, original=64, fast=16.0, slow=1.0),
                                     dict(factor=1.0, original=512, fast=32.0, slow=1.0),
                                     dict(factor=16.0, original=10 ** 6, fast=32.0, slow=2.0)])
def test_rotary_table(scaling):
    """Including a configuration whose blend range is empty (the slow end before the fast one)."""
    from types import SimpleNamespace

    from tokenweave_b200.layers.mixers import rope_table
    sizes = oracle.attn_layer(2, 8, 24, 8, 16, 16, None, base=300.0, scaling=scaling)["mixer"]
    rt = SimpleNamespace(rope_tables={}, max_positions=200, device="cpu")
    table, x = rope_table(rt, sizes["rot"]), torch.randn(24)
    assert rope_table(rt, dict(sizes["rot"])) is table and table.shape == (200, 24)
    for pos in (0, 1, 63, 199):
        cache = torch.zeros(1, 1, hops.latent_row(8, 24))
        p = torch.cat([torch.zeros(8), torch.ones(8), x]).view(1, -1)
        hops.latent_prep(p, 0, 8, torch.ones(8), torch.zeros(1, 8), 8, 8, torch.ones(8), 24, 24, table, i32([pos]), i32([0]),
                         cache, EPS)
        close(cache[0, 0, 8:], oracle.rotate(x.double(), pos, sizes["rot"]))


def test_norms_and_activation():
    y, w, wf, z = torch.randn(5, 24), torch.randn(24), torch.randn(24), torch.randn(5, 24) * 2
    x, xa = torch.randn(5, 24), torch.zeros(5, 24)
    want = x.double() + oracle.rms_unit(y.double(), EPS) * w
    got = x.clone()
    hops.postnorm_add_(y, got, w, EPS, xa)
    close(got, want)
    close(xa, want)
    hops.postnorm_add_(y, x, w, EPS, xa, wf)
    close(xa, oracle.rms_unit(want, EPS) * wf)
    W = {"act": torch.tensor([0.5, -1.0, 0.25, 0.75]).double(), "up": torch.eye(24).double(), "down": torch.eye(24).double()}
    close(hops.polynorm(z, W["act"].float(), EPS, torch.zeros(5, 24), 24), oracle.feed_forward(z.double(), W, EPS))
    for groups in (1, 3):
        got = hops.gated_group_norm(y, z, w, groups, EPS, torch.zeros(5, 24))
        close(got, oracle.grouped_norm(y.double() * oracle.silu(z.double()), groups, w.double(), EPS))


@pytest.mark.parametrize("taps", [1, 2, 4])
@pytest.mark.parametrize("cuts", [[9], [1] * 9, [2, 3, 2, 2], [8, 1]])
def test_convolution_and_recurrence_in_portions(taps, cuts):
    """A sequence cut in portions, its slot full of another sequence's leftovers at the start."""
    H, P, N, G = 4, 3, 5, 2
    ch, T = H * P + 2 * G * N, 9
    x, w, b = torch.randn(T, ch), torch.randn(taps, ch), torch.randn(ch)
    dt, bias, A, D = torch.randn(T, H), torch.randn(H), torch.randn(H) * 0.5, torch.randn(H)
    cst, st = torch.randn(3, taps - 1, ch), torch.randn(3, H, P, N)
    conv, y = torch.zeros(T, ch), torch.zeros(T, H * P)
    at = 0
    for n in cuts:
        rows = slice(at, at + n)
        meta = (i32([0, n]), i32([at + n]), i32([2]))
        hops.causal_conv(x[rows], w, b, cst, conv[rows], i32([0] * n), *meta, n == 1)
        hops.ssd_scan(conv[rows], dt[rows], bias, A, D, st, y[rows], i32([0]), *meta, G)
        at += n
    act = oracle.short_conv(x.double(), w.t().double(), b.double())
    close(conv, act)
    xs = act[:, :H * P].view(T, H, P)
    B, C = (act[:, H * P + k * G * N:H * P + (k + 1) * G * N].view(T, G, N)[:, [0, 0, 1, 1]] for k in (0, 1))
    want = oracle.state_space(xs, B, C, oracle.softplus(dt.double() + bias), A.double(), D.double())
    close(y, want.reshape(T, -1), 1e-4)


def test_state_slots():
    pool = StateSlotPool(2)
    a, b = pool.allocate(), pool.allocate()
    assert {a, b} == {0, 1} and pool.num_free == 0
    pool.release(a)
    with pytest.raises(AssertionError):
        pool.release(a)
    kv = KVCacheManager(8, 4, num_state_slots=2)
    reqs = [Request(str(i), [1] * 6, SamplingParams()) for i in range(3)]
    assert kv.allocate_slots(reqs[0], 6) and kv.allocate_slots(reqs[1], 6)
    held = reqs[0].state_slot
    assert not kv.allocate_slots(reqs[2], 4)                        # blocks are left, slots are not
    assert reqs[2].state_slot is None and not reqs[2].block_ids
    assert kv.allocate_slots(reqs[0], 8) and reqs[0].state_slot == held
    kv.free(reqs[0])
    assert reqs[0].state_slot is None and kv.allocate_slots(reqs[2], 4) and reqs[2].state_slot == held
    assert not kv.allocate_slots(Request("x", [1] * 40, SamplingParams()), 40) and kv.states.num_free == 0


def test_row_routing():
    """Every row is attended exactly once, long runs in tiles while their contexts fit, recurrences by run length."""
    from tokenweave_b200.models.hybrid import HybridDecoder
    from tokenweave_b200.parallel import state as pstate
    pstate.set_single_process(torch.device("cpu"))
    cfg = EngineArgs(model="tiny-sidisun", device="cpu", dtype="float32", max_num_batched_tokens=512,
                     max_model_len=512).create_engine_config()
    model = HybridDecoder(cfg.model, device="cpu")
    model.setup_runtime(512, cfg.tokenweave)
    model.tiles, model.rt.context_rows = True, 600
    q = [1, 64, 16, 40, 200, 20]
    kv = [300, 64, 30, 500, 400, 200]
    (tile_seq, tile_q0, tok_row, tok_seq, tok_kv), extra, host = model.plan_step(q, kv, list(range(6)), [-1] * 6)
    tiled = sorted(set(tile_seq))
    assert tiled == [1, 2, 4] and host == {"ctx_rows": 494, "ctx_max": 400}
    assert list(extra["ctx_begin"]) == [-1, 0, 64, -1, 94, -1] and list(extra["ctx_cu"]) == [0, 64, 94, 494]
    assert sorted(zip(tile_seq, tile_q0)) == [(1, 0), (2, 0), (4, 0), (4, 128)]
    start = np.cumsum([0] + q)
    rows = [(b, i) for b in (0, 3, 5) for i in range(q[b])]
    assert list(tok_row) == [start[b] + i for b, i in rows] and list(tok_seq) == [b for b, _ in rows]
    assert list(tok_kv) == [kv[b] - q[b] + i + 1 for b, i in rows]
    assert list(extra["scan_seqs"]) == [0] and list(extra["chunk_seqs"]) == [1, 2, 3, 4, 5]
    # under a window of 150 only the visible keys' tiles travel: the contexts of all long runs are short then
    model.expand_window = 150
    plan, extra, host = model.plan_step(q, kv, list(range(6)), [-1] * 6)
    assert sorted(set(plan[0])) == [1, 2, 4] and list(extra["ctx_first"]) == [0, 0, 0]      # (200 - 150 + 1 is in tile 0)
    model.expand_window = 60
    plan, extra, host = model.plan_step(q, kv, list(range(6)), [-1] * 6)
    assert sorted(set(plan[0])) == [1, 2, 4] and list(extra["ctx_first"]) == [0, 0, 128]    # (200 - 60 + 1 in tile 1)
    assert list(extra["ctx_cu"]) == [0, 64, 94, 366] and list(extra["ctx_begin"]) == [-1, 0, 64, -1, -34, -1]
    assert host == {"ctx_rows": 366, "ctx_max": 272}
    model.expand_window = 0
    model.rt.context_rows = 100                                      # the long context no longer fits
    assert sorted(set(model.plan_step(q, kv, list(range(6)), [-1] * 6)[0][0])) == [1, 2]
    plan, extra, _ = model.plan_step([1, 1], [5, 9], [1, 0], [-1] * 2)
    assert list(plan[2]) == [0, 1] and list(plan[4]) == [5, 9] and list(extra["state_slots"]) == [1, 0]

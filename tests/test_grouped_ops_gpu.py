"""Kernels of parallel blocks (grouped attention with its options, lightning attention, pair embeddings, sums and norms,
fused projections) against plain fp32 on the CPU, in bf16 and true fp32, sizes on and off the tile sizes."""
import numpy as np
import pytest
import torch

from tokenweave_b200 import ops
from tokenweave_b200.layers.attention import build_attention_metadata
from tokenweave_b200.ops import hybrid as hops
from tokenweave_b200.ops import reference_hybrid as ref

pytestmark = pytest.mark.gpu
DTYPES = [torch.bfloat16, torch.float32]
TOL = {torch.bfloat16: 8e-3, torch.float32: 2e-5}


def pad8(n):
    return (n + 7) // 8 * 8


def rnd(*shape, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape) * scale).to(dtype)


def heads_padded(T, parts, dtype):
    """Rows of heads padded to eight elements with zeros: parts = [(heads, size), ...]."""
    cols = []
    for n, d in parts:
        x = torch.zeros(T, n, pad8(d), dtype=dtype)
        x[..., :d] = rnd(T, n, d).to(dtype)
        cols.append(x.reshape(T, -1))
    return torch.cat(cols, 1)


def close(got, want, dtype, what="", scale=1.0):
    got, want = got.float().cpu(), want.float()
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-6)
    assert err < TOL[dtype] * scale, f"{what}: relative error {err:.2e}"


def meta_for(q_lens, kv_lens, page, device, tiles, seed=0, slots=None):
    """Metadata of a step over a shuffled block table, with every row routed to tiles or to single rows."""
    rng = np.random.default_rng(seed)
    B = len(q_lens)
    need = [(kv + page - 1) // page for kv in kv_lens]
    blocks = rng.permutation(np.arange(1, sum(need) + 1))
    table = np.zeros((B, max(need)), dtype=np.int32)
    at = 0
    for b, n in enumerate(need):
        table[b, :n] = blocks[at:at + n]
        at += n
    pos = np.concatenate([np.arange(kv - q, kv) for q, kv in zip(q_lens, kv_lens)])
    seq = np.repeat(np.arange(B), q_lens)
    slot = table[seq, pos // page] * page + pos % page
    tiled = [b for b in range(B) if tiles and q_lens[b] >= 16]
    row = np.flatnonzero(~np.isin(seq, tiled)).astype(np.int32)
    ts = [b for b in tiled for _ in range(0, q_lens[b], 128)]
    tq = [q0 for b in tiled for q0 in range(0, q_lens[b], 128)]
    plan = (ts, tq, row, seq[row], pos[row] + 1)
    extra = {"row_seq": seq, "state_slots": np.asarray(slots if slots is not None else range(B))}
    m = build_attention_metadata(q_lens, kv_lens, pos, slot, table, torch.device(device), plan=plan, extra=extra)
    return m, sum(need) + 1


STEPS = [([1, 1, 1], [1, 260, 700]), ([40, 1, 3, 130, 2], [40, 300, 3, 400, 65]), ([300], [300]), ([128, 17], [256, 513])]
HEADS = [(4, 2, 40, 24), (8, 8, 64, 48), (3, 1, 10, 13), (8, 2, 128, 128), (20, 1, 96, 72), (16, 2, 128, 64), (8, 1, 64, 120)]


@pytest.mark.parametrize("dtype", DTYPES, ids=["bf16", "fp32"])
@pytest.mark.parametrize("opts", ["plain", "bias+sink", "sink"])
@pytest.mark.parametrize("heads", HEADS)
@pytest.mark.parametrize("step", STEPS)
def test_grouped_attention(step, heads, opts, dtype):
    H, G, D, V = heads
    q_lens, kv_lens = step
    T = sum(q_lens)
    for page in (16, 64):
        tiles = hops.attention_tileable(dtype, pad8(D), pad8(V))
        mc, nb = meta_for(q_lens, kv_lens, page, "cpu", tiles)
        mg, _ = meta_for(q_lens, kv_lens, page, "cuda", tiles)
        q = heads_padded(T, [(H, D)], dtype) * 2
        kc = heads_padded(nb * page, [(G, D)], dtype).view(nb, page, G, -1)
        vc = heads_padded(nb * page, [(G, V)], dtype).view(nb, page, G, -1)
        slopes = torch.exp2(-8.0 * torch.arange(1, H + 1) / H) if "bias" in opts else None
        out = torch.zeros(T, H * pad8(V))
        args = (H, G, D ** -0.5, slopes, "sink" in opts, 0.7)
        ref.grouped_attention(q.float(), kc.float(), vc.float(), out, mc, *args)
        got = torch.full((T, H * pad8(V)), 9.0, dtype=dtype, device="cuda")
        dev = [x.cuda() if x is not None else None for x in (q, kc, vc, slopes)]
        hops.grouped_attention(dev[0], dev[1], dev[2], got, mg, H, G, D ** -0.5, dev[3], "sink" in opts, 0.7)
        ops.check_status()
        close(got, out, dtype, f"page {page}")


@pytest.mark.parametrize("dtype", DTYPES, ids=["bf16", "fp32"])
@pytest.mark.parametrize("bias", [False, True])
@pytest.mark.parametrize("where", ["prompt", "decoded"])
def test_every_single_key_is_seen(where, bias, dtype):
    """One key at a time stands out (first tokens, page and tile edges, the key before the query): its value comes back.
    Values are one-hot in the key's number, so that any other key shows."""
    H, G, D, V, page, n = 4, 2, 64, 64, 64, 300
    q_lens = [n] if where == "prompt" else [1]
    m, nb = meta_for(q_lens, [n], page, "cuda", dtype == torch.bfloat16)
    slopes = torch.exp2(-8.0 * torch.arange(1, H + 1) / H).cuda() if bias else None
    table = m.block_table[0].long()
    for key in (0, 1, 2, 63, 64, 127, 128, 129, 191, 192, 255, 256, 298, 299):
        k = torch.zeros(n, G, D)
        k[key, :, 0] = 30.0
        v = torch.zeros(n, G, V)
        v[key] = 3.0
        kc, vc = (torch.zeros(nb * page, G, x.shape[-1]) for x in (k, v))
        at = (table.cpu()[torch.arange(n) // page] * page + torch.arange(n) % page)
        kc[at], vc[at] = k, v
        q = torch.zeros(q_lens[0], H, D)
        q[..., 0] = 40.0
        out = torch.zeros(q_lens[0], H * V, dtype=dtype, device="cuda")
        to = lambda t: t.to(dtype).cuda()
        hops.grouped_attention(to(q).view(q_lens[0], -1), to(kc).view(nb, page, G, D), to(vc).view(nb, page, G, V), out, m, H,
                               G, 0.5, slopes, True, 1.0)
        ops.check_status()
        got = out.float().cpu().view(q_lens[0], H, V)
        assert (got[-1] - 3.0).abs().max() < 0.02, f"key {key} is not seen"
        if where == "prompt" and key > 0:
            assert got[:key].abs().max() < 1e-3, f"key {key} is seen before its time"


@pytest.mark.parametrize("dtype", DTYPES, ids=["bf16", "fp32"])
@pytest.mark.parametrize("norm", [None, "head", "whole"])
@pytest.mark.parametrize("taps", [None, 1, 2, 3, 5])
@pytest.mark.parametrize("heads", [(4, 2, 40, 24), (3, 1, 10, 13), (6, 2, 128, 64), (2, 1, 200, 72), (40, 8, 128, 128)])
def test_qkv_prep(heads, taps, norm, dtype):
    H, G, D, V = heads
    page = 16
    channels = H * pad8(D) + G * (pad8(D) + pad8(V))
    w = heads_padded(taps, [(H, D), (G, D), (G, V)], dtype) if taps else None
    n = (H, G) if norm == "whole" else (1, 1)
    wq, wk = ((1 + 0.3 * heads_padded(1, [(i, D)], torch.float32)).to(dtype).view(-1) if norm else None for i in n)
    # two steps in a row: portions and single tokens beside one another, then single tokens only
    state = rnd(7, max(0, (taps or 1) - 1), channels, dtype=dtype)
    state_g = state.cuda()
    caches = None
    for q_lens, kv_lens in (([5, 1, 2, 30], [5, 9, 64, 30]), ([1, 1, 1, 1], [6, 10, 65, 31])):
        T = sum(q_lens)
        slots = [6, 0, 3, 2]
        mc, nb = meta_for(q_lens, [96] * 4, page, "cpu", False, slots=slots)     # (a table long enough for both steps)
        pos = np.concatenate([np.arange(kv - q, kv) for q, kv in zip(q_lens, kv_lens)])
        seq = np.repeat(np.arange(4), q_lens)
        table = mc.block_table.numpy()
        slot = table[seq, pos // page] * page + pos % page
        build = lambda dev: build_attention_metadata(
            q_lens, kv_lens, pos, slot, table, torch.device(dev), plan=([], [], [], [], []),
            extra={"row_seq": seq, "state_slots": np.asarray(slots)})
        mc, mg = build("cpu"), build("cuda")
        if caches is None:
            caches = [torch.zeros(nb, page, G, pad8(d), dtype=dtype) for d in (D, V)]
            caches_g = [c.cuda() for c in caches]
        p = heads_padded(T, [(H, D), (G, D), (G, V)], dtype)
        q, qg = torch.zeros(T, H * pad8(D), dtype=dtype), torch.zeros(T, H * pad8(D), dtype=dtype, device="cuda")
        cuda = lambda x: x.cuda() if x is not None else None
        args = lambda f: (norm, f(wq), f(wk), 1e-5, 0.4, 7)
        same = lambda x: x
        hops.qkv_prep(p, H, G, D, V, q, *caches, mc, w, state if (taps or 0) > 1 else None, *args(same))
        hops.qkv_prep(p.cuda(), H, G, D, V, qg, *caches_g, mg, cuda(w), state_g if (taps or 0) > 1 else None, *args(cuda))
        close(qg, q, dtype, "queries")
        close(caches_g[0], caches[0], dtype, "keys")
        close(caches_g[1], caches[1], dtype, "values")
        if (taps or 0) > 1:
            close(state_g, state, dtype, "state")


@pytest.mark.parametrize("dtype", DTYPES, ids=["bf16", "fp32"])
@pytest.mark.parametrize("sizes", [(3, 24, 16), (2, 40, 72), (4, 64, 128), (2, 136, 64), (3, 8, 8), (2, 300, 24)])
def test_lightning_recurrence(sizes, dtype):
    H, N, P = sizes
    decay = torch.tensor([0.999, 0.3, 1.0, 0.0][:H])
    q_lens, kv_lens = [1, 130, 300, 16, 5, 40], [1, 130, 500, 16, 9, 41]
    T, B = sum(q_lens), len(q_lens)
    cu = torch.tensor(np.concatenate([[0], np.cumsum(q_lens)]), dtype=torch.int32)
    kv, slots = torch.tensor(kv_lens, dtype=torch.int32), torch.tensor([3, 0, 5, 1, 2, 4], dtype=torch.int32)
    p = rnd(T, H * (P + 2 * N) + 8, dtype=dtype, scale=0.5)
    state = rnd(6, H, P, N)
    y, want_state = torch.zeros(T, H * P), state.clone()
    seqs = torch.arange(B, dtype=torch.int32)
    ref.decay_scan(p.float(), decay, want_state, y, seqs, cu, kv, slots)
    forms = [hops.decay_scan]
    if hops.ssd_chunkable(dtype, P, N):
        forms += [hops.decay_chunk, lambda *a: hops.decay_chunk(*a, form=1)]
    for run in forms:
        st, out = state.cuda(), torch.zeros(T, H * P, dtype=dtype, device="cuda")
        run(p.cuda(), decay.cuda(), st, out, seqs.cuda(), cu.cuda(), kv.cuda(), slots.cuda())
        ops.check_status()
        close(out, y, dtype, "outputs")
        close(st, want_state, torch.float32, "state", 20.0 if dtype == torch.bfloat16 else 1.0)


@pytest.mark.parametrize("dtype", DTYPES, ids=["bf16", "fp32"])
@pytest.mark.parametrize("width", [40, 45, 1000, 4096, 11008])
def test_embedding_sum_and_norm(width, dtype):
    vocab, spec = 83, {"buckets": 61, "mul_prev": 1000003, "mul_cur": 777}
    w8 = pad8(width)
    q_lens, kv_lens = [3, 1, 1, 20], [3, 1, 9, 30]
    T = sum(q_lens)
    m = {d: meta_for(q_lens, kv_lens, 16, d, False)[0] for d in ("cpu", "cuda")}
    for d in m:
        m[d].extra["prev_token"] = torch.tensor([-1, -1, 5, 82], dtype=torch.int32, device=d)
    ids = torch.randint(0, vocab, (T,), dtype=torch.int32)
    table, pairs = torch.zeros(vocab, w8, dtype=dtype), torch.zeros(62, w8, dtype=dtype)
    table[:, :width], pairs[:, :width] = rnd(vocab, width).to(dtype), rnd(62, width).to(dtype)
    w, y = rnd(width, dtype=dtype), rnd(T, w8, dtype=dtype)
    res = {}
    for d in ("cpu", "cuda"):
        x32, first = (torch.zeros(T, w8, device=d) for _ in range(2))
        xa, xb = (torch.zeros(T, w8, dtype=dtype, device=d) for _ in range(2))
        to = lambda t: t.to(d)
        hops.embed_norm(to(ids), to(table), to(pairs), spec, m[d], x32, first, to(w), 1e-3, xa)
        kept = x32.clone()
        hops.add_prenorm_(to(y), x32, first, to(w), 1e-3, xb)
        hops.add_prenorm_(to(y), x32, None, to(w), 1e-3, xb)
        res[d] = [t.cpu() for t in (kept, first, xa, x32, xb)]
    for a, b, name in zip(res["cuda"], res["cpu"], ("stream", "first", "normed", "sum", "normed sum")):
        close(a, b, dtype if "normed" in name else torch.float32, name)
    rows = ref.pair_rows(ids, m["cpu"].extra["row_seq"], m["cpu"].cu_q, m["cpu"].extra["prev_token"], spec)
    want = [61, (int(ids[0]) * 1000003 + int(ids[1]) * 777) % 61]
    assert rows[:2].tolist() == want and rows[3] == 61 and rows[4] == (5 * 1000003 + int(ids[4]) * 777) % 61
    assert torch.equal(res["cuda"][0][:, :width], (table.float()[ids.long()] + pairs.float()[rows])[:, :width])


@pytest.mark.parametrize("dtype", DTYPES, ids=["bf16", "fp32"])
@pytest.mark.parametrize("sizes", [(3, 24), (6, 61), (32, 128)])
def test_norm_gate(sizes, dtype):
    H, V = sizes
    T, C = 19, H * pad8(V)
    y, g, w = (heads_padded(n, [(H, V)], dtype) for n in (T, T, 1))
    out = torch.zeros(T, C, dtype=dtype)
    ref.norm_gate(y, g, w.view(-1), H * V, 1e-5, -0.6, out)
    got = torch.zeros(T, C + 16, dtype=dtype, device="cuda")
    hops.norm_gate(y.cuda(), g.cuda(), w.view(-1).cuda(), H * V, 1e-5, -0.6, got[:, 8:8 + C])
    close(got[:, 8:8 + C], out, dtype)
    assert got[:, :8].abs().max() == 0 and got[:, 8 + C:].abs().max() == 0


@pytest.mark.parametrize("dtype", DTYPES, ids=["bf16", "fp32"])
@pytest.mark.parametrize("shape", [(1, 48, 80), (37, 64, 208), (300, 256, 1040), (2100, 512, 4096)])
def test_fused_projections(shape, dtype):
    """silu on a range of columns that starts and ends inside tiles, behind a bias; the gated product."""
    T, K, N = shape
    x, w, b = rnd(T, K, dtype=dtype), rnd(N, K, dtype=dtype, scale=K ** -0.5), rnd(N, dtype=dtype)
    for lo, hi in ((8, N - 16), (N // 3 // 8 * 8, N // 2 // 8 * 8), (0, N)):
        z = x.float() @ w.float().t() + b.float()
        z[:, lo:hi] = torch.nn.functional.silu(z[:, lo:hi])
        out = torch.zeros(T, N, dtype=dtype, device="cuda")
        hops.projection(x.cuda(), w.cuda(), b.cuda(), (lo, hi), out)
        ops.check_status()
        close(out, z, dtype, f"silu on [{lo}, {hi})")
    for act in ("silu", "gelu_tanh"):
        want = torch.zeros(T, N // 2)
        w[:N // 2] *= 3                                  # gates far into both tails
        ref.gated_product(x.float(), w.float(), act, want)
        out = torch.zeros(T, N // 2 + 24, dtype=dtype, device="cuda")
        tmp = torch.zeros(T, N, dtype=dtype, device="cuda")
        hops.gated_product(x.cuda(), w.cuda(), act, out[:, 8:8 + N // 2], tmp)
        ops.check_status()
        close(out[:, 8:8 + N // 2], want, dtype, act)
        assert out[:, :8].abs().max() == 0 and out[:, 8 + N // 2:].abs().max() == 0

"""Kernels of windowed attention with kept first keys, latent attention with a window and a sink, rotation of neighbouring
pairs, hyper-connections and routed feed-forwards against plain fp32 on the CPU, in bf16 and true fp32, sizes on and off the
tile sizes."""
import math

import numpy as np
import pytest
import torch

from test_grouped_ops_gpu import HEADS, STEPS, close, heads_padded, meta_for, pad8, rnd
from tokenweave_b200 import ops
from tokenweave_b200.ops import hybrid as hops
from tokenweave_b200.ops import reference
from tokenweave_b200.ops import reference_hybrid as ref

pytestmark = pytest.mark.gpu
DTYPES = [torch.bfloat16, torch.float32]
IDS = ["bf16", "fp32"]


@pytest.fixture(autouse=True)
def _status_clean():
    ops.reset_status()
    yield
    ops.check_status()


def i32(x):
    return torch.as_tensor(x, dtype=torch.int32)


# ---- grouped attention ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("window,keep", [(1, 0), (37, 4), (128, 0), (129, 3), (200, 130), (5000, 2)])
@pytest.mark.parametrize("heads", HEADS)
def test_windowed_attention(heads, window, keep, dtype):
    H, G, D, V = heads
    for i, (q_lens, kv_lens) in enumerate(STEPS):
        T, page = sum(q_lens), (16, 64)[(i + window) % 2]
        tiles = hops.attention_tileable(dtype, pad8(D), pad8(V))
        mc, nb = meta_for(q_lens, kv_lens, page, "cpu", tiles)
        mg, _ = meta_for(q_lens, kv_lens, page, "cuda", tiles)
        q = heads_padded(T, [(H, D)], dtype) * 2
        kc = heads_padded(nb * page, [(G, D)], dtype).view(nb, page, G, -1)
        vc = heads_padded(nb * page, [(G, V)], dtype).view(nb, page, G, -1)
        out = torch.zeros(T, H * pad8(V))
        ref.grouped_attention(q.float(), kc.float(), vc.float(), out, mc, H, G, D ** -0.5, None, False, 1.0, window, keep)
        got = torch.full((T, H * pad8(V)), 9.0, dtype=dtype, device="cuda")
        hops.grouped_attention(q.cuda(), kc.cuda(), vc.cuda(), got, mg, H, G, D ** -0.5, None, False, 1.0, window=window,
                               keep=keep)
        close(got, out, dtype, f"{q_lens}, page {page}")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("options", ["bias", "sink", "simt"])
def test_windows_beside_the_other_options(options, dtype):
    """Rows attended alone take a window together with a distance bias; a sink goes with every form."""
    H, G, D, V, page = 6, 2, 40, 24, 16
    bias = options == "bias"
    for q_lens, kv_lens in STEPS:
        T = sum(q_lens)
        tiles = dtype == torch.bfloat16 and options == "sink"
        (mc, nb), (mg, _) = (meta_for(q_lens, kv_lens, page, d, tiles) for d in ("cpu", "cuda"))
        q, kc, vc = heads_padded(T, [(H, D)], dtype), *(heads_padded(nb * page, [(G, n)], dtype).view(nb, page, G, -1) for n in (D, V))
        slopes = torch.exp2(-8.0 * torch.arange(1, H + 1) / H) if bias else None
        out, got = torch.zeros(T, H * V), torch.zeros(T, H * V, dtype=dtype, device="cuda")
        ref.grouped_attention(q.float(), kc.float(), vc.float(), out, mc, H, G, 0.2, slopes, True, 0.5, 70, 3)
        hops.grouped_attention(q.cuda(), kc.cuda(), vc.cuda(), got, mg, H, G, 0.2, slopes.cuda() if bias else None, True, 0.5,
                               kernel="simt" if options == "simt" else None, window=70, keep=3)
        close(got, out, dtype, str(q_lens))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("splits", ["planned", "many"])
@pytest.mark.parametrize("window,keep", [(60, 0), (128, 4), (129, 0), (203, 129), (300, 1)])
def test_every_key_is_seen_or_not(window, keep, splits, dtype):
    """One key at a time stands out: the prompt's rows and a decoded row see it exactly when the mask says so."""
    H, G, D, V, page, n = 4, 2, 64, 64, 64, 400
    for q_len in (n, 1):
        m, nb = meta_for([q_len], [n], page, "cuda", dtype == torch.bfloat16)
        if splits == "many":
            m.max_kv_len = 100 * n                   # more splits than there are tiles
        at = (m.block_table[0].cpu().long()[torch.arange(n) // page] * page + torch.arange(n) % page)
        for key in sorted({0, 1, keep - 1, keep, 127, 128, 255, n - window - 1, n - window, n - window + 1, n - 2, n - 1} & set(range(n))):
            kc, vc = torch.zeros(nb * page, G, D), torch.zeros(nb * page, G, V)
            kc[at[key], :, 0], vc[at[key]] = 30.0, 3.0
            q = torch.zeros(q_len, H, D)
            q[..., 0] = 40.0
            out = torch.zeros(q_len, H * V, dtype=dtype, device="cuda")
            to = lambda t: t.to(dtype).cuda()
            hops.grouped_attention(to(q).view(q_len, -1), to(kc).view(nb, page, G, D), to(vc).view(nb, page, G, V), out, m, H,
                                   G, 0.5, None, False, 1.0, window=window, keep=keep)
            i = torch.arange(n - q_len, n)
            sees = (key <= i) & ((i - key < window) | (key < keep))
            got = out.float().cpu().view(q_len, H, V)
            assert (got - 3.0 * sees[:, None, None]).abs().max() < 0.02, f"key {key} of {q_len} queries"


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("norm", [None, "head"])
@pytest.mark.parametrize("taps", [None, 3])
@pytest.mark.parametrize("heads,dims", [((4, 2, 40, 24), 16), ((3, 1, 10, 13), 6), ((8, 2, 128, 128), 128), ((2, 1, 200, 72), 44),
                                        ((40, 8, 128, 64), 64), ((5, 1, 16, 8), 2)])
def test_rotation_in_qkv_prep(heads, dims, taps, norm, dtype):
    H, G, D, V = heads
    page, q_lens, kv_lens = 16, [5, 1, 2, 30], [5, 9, 64, 300]
    T, channels = sum(q_lens), H * pad8(D) + G * (pad8(D) + pad8(V))
    (mc, nb), (mg, _) = (meta_for(q_lens, kv_lens, page, d, False, slots=[3, 0, 1, 2]) for d in ("cpu", "cuda"))
    table = reference.build_cos_sin_cache(dims, 300, 100.0)
    p = heads_padded(T, [(H, D), (G, D), (G, V)], dtype)
    w = heads_padded(taps, [(H, D), (G, D), (G, V)], dtype) if taps else None
    wq, wk = ((1 + 0.3 * heads_padded(1, [(1, D)], torch.float32)).to(dtype).view(-1) if norm else None for _ in "qk")
    res = {}
    for d, m in (("cpu", mc), ("cuda", mg)):
        to = lambda t: t.to(d) if t is not None else None
        q = torch.zeros(T, H * pad8(D), dtype=dtype, device=d)
        caches = [torch.zeros(nb, page, G, pad8(n), dtype=dtype, device=d) for n in (D, V)]
        state = torch.ones(4, 2, channels, dtype=dtype, device=d) if taps else None
        hops.qkv_prep(to(p), H, G, D, V, q, *caches, m, to(w), state, norm, to(wq), to(wk), 1e-5, 0.3, 5, to(table))
        res[d] = [t.cpu() for t in (q, *caches)]
    for got, want, name in zip(res["cuda"], res["cpu"], ("queries", "keys", "values")):
        close(got, want, dtype, name)


# ---- latent attention --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kernel,dtype", [("simt", torch.float32), ("simt", torch.bfloat16), ("tc", torch.bfloat16)])
@pytest.mark.parametrize("window", [1, 50, 128, 129, 300])
@pytest.mark.parametrize("heads,kv_rank,rot,page", [(3, 40, 16, 8), (16, 128, 32, 64), (20, 200, 24, 32), (40, 512, 64, 128)])
def test_windowed_latent_attention(kernel, dtype, heads, kv_rank, rot, page, window):
    from test_hybrid_ops_gpu import paged
    lens = [1, 7, page + 1, 127, 128, 129, 400, 1500]
    row = hops.latent_row(kv_rank, rot)
    cache, bt = paged(lens, page, row, dtype)
    n, scale = len(lens), 1.5 * row ** -0.5
    qa, sink = rnd(n, heads, row, dtype=dtype), rnd(heads, scale=3.0)
    tok_seq, tok_kv = i32(range(n)), i32(lens)
    out = torch.empty(n, heads, kv_rank, dtype=dtype, device="cuda")
    for s in (None, sink):
        want = ref.latent_attention(qa, cache, tok_seq, tok_kv, bt, kv_rank, scale, window, s)
        for max_len in (max(lens), 100 * max(lens)):
            hops.latent_attention(qa.cuda(), cache.cuda(), tok_seq.cuda(), tok_kv.cuda(), n, bt.cuda(), kv_rank, scale, out,
                                  max_len, kernel=kernel, window=window, sink=None if s is None else s.cuda())
            close(out, want, dtype)


@pytest.mark.parametrize("window", [0, 1, 60, 128, 129, 400])
@pytest.mark.parametrize("heads,dim,rot,vdim", [(3, 40, 16, 24), (2, 64, 32, 64), (4, 128, 64, 128), (2, 72, 8, 104),
                                                (2, 136, 32, 64)])
@pytest.mark.parametrize("q_lens,kv_lens", [([300], [300]), ([17, 128, 64], [40, 1000, 64]), ([2, 130], [130, 131])])
def test_windowed_latent_prefill(heads, dim, rot, vdim, window, q_lens, kv_lens):
    """Contexts begin with the first visible key's tile."""
    first = [max(0, m - n - window + 1) // 128 * 128 if window else 0 for n, m in zip(q_lens, kv_lens)]
    held = [m - f for m, f in zip(kv_lens, first)]
    T, rows = sum(q_lens), sum(held)
    q, kv = rnd(T, heads * (dim + rot), dtype=torch.bfloat16), rnd(rows, heads * (dim + vdim), dtype=torch.bfloat16)
    lat, sink = rnd(rows, 16 + rot, dtype=torch.bfloat16), rnd(heads, scale=2.0)
    scale = 2.0 * (dim + rot) ** -0.5
    cu = np.concatenate([[0], np.cumsum(q_lens)]).tolist()
    at = np.concatenate([[0], np.cumsum(held)]).tolist()
    tiles = [(b, q0) for b, n in enumerate(q_lens) for q0 in range(0, n, 128)]
    want = {s: torch.zeros(T, heads * vdim) for s in (False, True)}
    for b, (n, m) in enumerate(zip(q_lens, held)):
        here = slice(at[b], at[b] + m)
        k = torch.cat([kv[here, :heads * dim].float().view(m, heads, dim), lat[here, None, 16:].float().expand(m, heads, rot)], -1)
        v = kv[here, heads * dim:].float().view(m, heads, vdim)
        s = torch.einsum("qhd,khd->hqk", q[cu[b]:cu[b + 1]].float().view(n, heads, dim + rot), k) * scale
        dist = torch.arange(m - n, m)[:, None] - torch.arange(m)[None]
        s = s.masked_fill((dist < 0) | ((dist >= window) if window else False), -math.inf)
        for with_sink in (False, True):
            x = torch.cat([s, sink[:, None, None].expand(heads, n, 1)], -1) if with_sink else s
            want[with_sink][cu[b]:cu[b + 1]] = torch.einsum("hqk,khd->qhd", x.softmax(-1)[..., :m], v).reshape(n, -1)
    g = lambda t: i32(t).cuda()
    for with_sink in (False, True):
        out = torch.zeros(T, heads * vdim, dtype=torch.bfloat16, device="cuda")
        hops.latent_prefill(q.cuda(), kv.cuda(), lat.cuda(), 16, rows, g([a - f for a, f in zip(at, first)]), out, None, g(cu),
                            g(kv_lens), g([b for b, _ in tiles]), g([q0 for _, q0 in tiles]), len(tiles), heads, dim, rot, vdim,
                            scale, window, sink.cuda() if with_sink else None)
        ops.check_status()
        close(out, want[with_sink], torch.bfloat16, f"sink {with_sink}")


def test_gather_from_a_key_on():
    from test_hybrid_ops_gpu import paged
    lens, page, row = [5, 330, 64, 33], 32, 24
    cache, bt = paged(lens, page, row, torch.bfloat16)
    seqs, first = [3, 1], [0, 128]
    out = torch.zeros(235, row, dtype=torch.bfloat16, device="cuda")
    hops.latent_gather(cache.cuda(), i32(seqs).cuda(), i32([0, 33, 235]).cuda(), 202, bt.cuda(), out, i32(first).cuda())
    want = torch.cat([cache[bt[s].long()].reshape(-1, row)[f:lens[s]] for s, f in zip(seqs, first)])
    assert torch.equal(out.cpu(), want)


# ---- hyper-connections --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 7, 16])
@pytest.mark.parametrize("T,W", [(1, 40), (5, 45), (33, 1000), (3, 4096), (2, 5000), (2, 11008)])
def test_streams(T, W, streams, dtype):
    w8, vocab = pad8(W), 31
    table = torch.zeros(vocab, w8, dtype=dtype)
    table[:, :W] = rnd(vocab, W).to(dtype)
    ids = torch.randint(0, vocab, (T,), dtype=torch.int32)
    y, w = rnd(T, w8, dtype=dtype), rnd(W, dtype=dtype, scale=0.3)
    hc = {"in": rnd(streams), "out": rnd(streams), "mix": rnd(streams, streams)}
    nxt, res = rnd(streams), {}
    for d in ("cpu", "cuda"):
        to = lambda t: t.to(d)
        x = torch.zeros(T, streams, w8, device=d)
        a, b, c = (torch.zeros(T, w8, dtype=dtype, device=d) for _ in range(3))
        h = {k: to(v) for k, v in hc.items()}
        hops.embed_streams(to(ids), to(table), x, h["in"], to(w), 1.0, 1e-4, a)
        start = x.clone()
        hops.streams_step(to(y), x, h, 0.3, to(nxt), to(w), 1.0, 1e-4, b, first=True)
        hops.streams_step(to(y), x, h, 0.3, to(nxt), to(w), 1.0, 1e-4, b)
        kept = x.clone()
        hops.streams_step(to(y), x, h, 0.3, None, to(w), 1.0, 1e-4, c)
        assert torch.equal(x, kept)                   # behind the last sublayer the streams stay
        res[d] = [t.cpu() for t in (start, x, a, b, c)]
    for got, want, name in zip(res["cuda"], res["cpu"], ("embedded", "streams", "first", "next", "last")):
        close(got, want, torch.float32 if name in ("embedded", "streams") else dtype, name)
    assert res["cuda"][1][..., W:].abs().sum() == 0 and res["cuda"][3][:, W:].abs().sum() == 0


# ---- feed-forwards ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("T,H,E,top,gates", [(1, 40, 5, 3, 1), (37, 48, 16, 4, 0), (300, 256, 64, 8, 1), (5000, 64, 8, 2, 1),
                                             (130, 4096, 33, 5, 2), (9, 1000, 256, 32, 8), (20, 16, 1, 1, 1)])
def test_router(T, H, E, top, gates, dtype):
    x, w, corr = rnd(T, H, dtype=dtype), rnd(E + gates, H, dtype=dtype, scale=2 * H ** -0.5), torch.rand(E) * 0.3
    for c in (corr, None):
        got_w, got_i, got_g = ops.moe_route(x.cuda(), w.cuda(), E, top, None if c is None else c.cuda(), 1e-20)
        _, _, g = reference.moe_route(x, w, E, top, c, 1e-20)
        close(got_g, g, torch.float32, "gates", 10.0) if gates else None
        scores = torch.softmax(x.double() @ w[:E].double().t(), -1)
        choice = scores if c is None else scores + c
        ids = got_i.cpu().long()
        assert all(len(set(r)) == top for r in ids.tolist())
        # the chosen ones are the largest (but for near ties), in falling order, and the weights are their scores' shares
        picked = choice.gather(1, ids)
        best = choice.topk(top, -1).values
        assert (picked - best).abs().max() < 1e-5
        share = scores.gather(1, ids)
        close(got_w, (share / share.sum(-1, keepdim=True)).float(), torch.float32, "weights", 5.0)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("shape", [(1, 48, 80), (37, 64, 208), (300, 256, 1040), (2100, 512, 4096)])
def test_activations_of_products(shape, dtype):
    T, K, N = shape
    x, w = rnd(T, K, dtype=dtype), rnd(N, K, dtype=dtype, scale=K ** -0.5)
    z = x.float() @ w.float().t()
    for lo, hi in ((0, N), (8, N - 16)):
        want = z.clone()
        want[:, lo:hi] = torch.relu(want[:, lo:hi]) ** 2
        out = torch.zeros(T, N, dtype=dtype, device="cuda")
        hops.projection(x.cuda(), w.cuda(), None, (lo, hi), out, "relu2")
        close(out, want, dtype, f"relu2 on [{lo}, {hi})")
    for limit in (0.4, 2.0):
        want = torch.zeros(T, N // 2)
        ref.gated_product(x.float(), w.float(), ("clamped", limit, 1.702), want)
        out, tmp = (torch.zeros(T, n, dtype=dtype, device="cuda") for n in (N // 2, N))
        hops.gated_product(x.cuda(), w.cuda(), ("clamped", limit, 1.702), out, tmp)
        close(out, want, dtype, f"limit {limit}")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("T,width,E,top,ff,shared", [(1, 40, 5, 3, 11, 7), (200, 45, 16, 4, 64, None), (90, 256, 64, 8, 96, 128),
                                                     (3000, 128, 4, 2, 136, 72), (1500, 64, 3, 3, 24, 40)])
def test_routed_feed_forward(T, width, E, top, ff, shared, dtype):
    """The layer on the GPU against the same layer's plain path, rows sorted into groups of 128 and of 256."""
    from types import SimpleNamespace

    from tokenweave_b200.layers.mixers import RoutedMLP
    sizes = dict(experts=E, top=top, ff=ff, act=("clamped", 1.1, 1.702), sum_eps=1e-20,
                 shared=dict(ff=shared, act=("clamped", 0.8, 1.702)) if shared else None)
    w8, res = pad8(width), {}
    x = torch.zeros(T, w8, dtype=dtype)
    x[:, :width] = rnd(T, width).to(dtype)
    weights = None
    for d in ("cpu", "cuda"):
        layer = RoutedMLP(sizes, width, 1e-5, dtype=dtype, device=d)
        targets = layer.tensor_targets()
        if weights is None:
            weights = {k: (torch.rand(s) if k == "correction" else rnd(*s, scale=2 * s[-1] ** -0.5)).to(torch.bfloat16)
                       for k, (s, _) in targets.items()}
        for k, (_, put) in targets.items():
            put(weights[k])
        made = {}

        def buffer(name, rows, cols):
            key = (name, cols)
            if key not in made or made[key].shape[0] < rows:
                made[key] = torch.zeros(rows, cols, dtype=dtype, device=d)
            return made[key][:rows]
        rt = SimpleNamespace(max_tokens=T, tables={}, buffer=buffer)
        layer.bind_runtime(rt)
        out = torch.full((T, w8), 9.0, dtype=dtype, device=d)
        layer(x.to(d), rt, out)
        res[d] = out.cpu()
    assert res["cuda"][:, width:].abs().sum() == 0
    got, want = res["cuda"].float(), res["cpu"].float()
    off = (got - want).abs().amax(-1) / want.abs().max()
    limit = 1.5e-2 if dtype == torch.bfloat16 else 2e-5
    # (a token whose choice is nearly tied may take another expert)
    assert (off > limit).float().mean() <= 0.01, f"{(off > limit).sum()} of {T} rows are off by up to {off.max():.2e}"

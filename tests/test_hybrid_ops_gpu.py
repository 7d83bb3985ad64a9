"""Kernels of the hybrid operators (``ops/hybrid.py``) against plain fp32 PyTorch on the CPU: bf16 and fp32 storage, sizes
that are not multiples of anything, and the tensor-core forms against the same references."""
import functools
import math

import pytest
import torch

pytestmark = pytest.mark.gpu
if torch.cuda.is_available():
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    from tokenweave_b200.ops import reference, reference_hybrid as ref

DEV = "cuda"
DTYPES = [torch.bfloat16, torch.float32]


def rnd(*shape, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape) * scale).to(dtype)


def tol(dtype):
    return dict(atol=2e-2, rtol=2e-2) if dtype == torch.bfloat16 else dict(atol=2e-5, rtol=2e-5)


def i32(x):
    return torch.as_tensor(x, dtype=torch.int32)


@pytest.fixture(autouse=True)
def _status_clean():
    ops.reset_status()
    yield
    ops.check_status()


@pytest.mark.parametrize("M,N,K", [(1, 7, 5), (65, 130, 33), (300, 64, 200)])
def test_gemm_f32(M, N, K):
    a, w, b = rnd(M, K), rnd(N, K), rnd(N)
    out = ops.gemm(a.to(DEV), w.to(DEV), bias=b.to(DEV))
    want = (a.double() @ w.double().t() + b.double()).float()
    torch.testing.assert_close(out.cpu(), want, atol=1e-4, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H", [(1, 24), (5, 203), (40, 1024), (3, 9000)])
def test_residual_rows(dtype, T, H):
    ld = (H + 7) // 8 * 8
    table, ids = rnd(50, ld, dtype=dtype), i32(torch.randint(0, 50, (T,)))
    x = [torch.zeros(T, ld), torch.zeros(T, ld, dtype=dtype)]
    g = [t.to(DEV) for t in x]
    ref.embed_residual(ids, table, *x, H)
    hops.embed_residual(ids.to(DEV), table.to(DEV), *g, H)
    assert torch.equal(g[0].cpu(), x[0]) and torch.equal(g[1].cpu(), x[1])
    y, w, wf = rnd(T, ld, dtype=dtype, scale=3), rnd(H, dtype=dtype), rnd(H, dtype=dtype)
    for final in (None, wf):
        ref.postnorm_add_(y, x[0], w, 1e-5, x[1], final)
        hops.postnorm_add_(y.to(DEV), g[0], w.to(DEV), 1e-5, g[1], None if final is None else final.to(DEV))
        torch.testing.assert_close(g[0].cpu(), x[0], atol=1e-5, rtol=1e-5)
        torch.testing.assert_close(g[1].cpu(), x[1], **tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,C,groups", [(3, 40, 1), (7, 210, 3), (33, 2048, 8), (2, 9000, 2)])
def test_activation_rows(dtype, T, C, groups):
    ld = (C + 7) // 8 * 8
    z, y, w = rnd(T, ld, dtype=dtype, scale=2), rnd(T, ld, dtype=dtype), rnd(C, dtype=dtype)
    coef = torch.tensor([0.5, -0.75, 0.25, 0.125]).to(dtype)
    out = torch.zeros(T, ld, dtype=dtype, device=DEV)
    hops.polynorm(z.to(DEV), coef.to(DEV), 1e-5, out, C)
    torch.testing.assert_close(out[:, :C].cpu(), ref.polynorm(z[:, :C], coef, 1e-5), **tol(dtype))
    hops.gated_group_norm(y.to(DEV), z.to(DEV), w.to(DEV), groups, 1e-5, out)
    torch.testing.assert_close(out[:, :C].cpu(), ref.gated_group_norm(y[:, :C], z[:, :C], w, groups, 1e-5), **tol(dtype))


def paged(lens, page, row, dtype, spare=3, scale=1.0):
    """A latent cache with shuffled pages: (cache, block table)."""
    need = [(n + page - 1) // page for n in lens]
    order = torch.randperm(sum(need) + spare)[: sum(need)] + 1
    bt = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
    k = 0
    for b, n in enumerate(need):
        bt[b, :n] = order[k:k + n].int()
        k += n
    cache = rnd(sum(need) + spare + 1, page, row, dtype=dtype, scale=scale)
    return cache, bt


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,kv_rank,rot,rot_dims", [(24, 40, 16, 16), (50, 37, 12, 8), (1536, 512, 64, 64), (3001, 600, 20, 20)])
def test_latent_prep_and_absorb(dtype, q_rank, kv_rank, rot, rot_dims):
    T, heads, dim, page = 9, 3, 20, 8
    p8 = lambda n: (n + 7) // 8 * 8
    kv_off = p8(q_rank)
    p = rnd(T, kv_off + p8(kv_rank + rot), dtype=dtype)
    wq, wkv = rnd(q_rank, dtype=dtype), rnd(kv_rank, dtype=dtype)
    cs = reference.build_cos_sin_cache(rot_dims, 300, 10000.0)
    pos = i32(torch.randint(0, 300, (T,)))
    slots = i32(torch.randperm(T * 4)[:T])
    slots[4] = -1
    row = hops.latent_row(kv_rank, rot)
    cq, cache = torch.zeros(T, p8(q_rank), dtype=dtype), rnd(T * 4 // page + 1, page, row, dtype=dtype)
    gq, gc = cq.to(DEV), cache.to(DEV)
    ref.latent_prep(p, 0, q_rank, wq, cq, kv_off, kv_rank, wkv, rot, rot_dims, cs, pos, slots, cache, 1e-5)
    hops.latent_prep(p.to(DEV), 0, q_rank, wq.to(DEV), gq, kv_off, kv_rank, wkv.to(DEV), rot, rot_dims, cs.to(DEV),
                     pos.to(DEV), slots.to(DEV), gc, 1e-5)
    torch.testing.assert_close(gq.cpu(), cq, **tol(dtype))
    torch.testing.assert_close(gc.cpu(), cache, **tol(dtype))
    q = rnd(T, p8(heads * (dim + rot)), dtype=dtype)
    ukt = rnd(heads, kv_rank, p8(dim), dtype=dtype, scale=dim ** -0.5)
    rows = i32([7, 0, 3, 8])
    qa = torch.full((4, heads, row), 9.0, dtype=dtype, device=DEV)
    hops.latent_absorb(q.to(DEV), rows.to(DEV), ukt.to(DEV), heads, dim, rot, rot_dims, kv_rank, cs.to(DEV), pos.to(DEV), qa)
    want = ref.latent_absorb(q, rows, ukt, heads, dim, rot, rot_dims, kv_rank, cs, pos, row)
    torch.testing.assert_close(qa.cpu(), want, **tol(dtype))
    vdim = 28
    o, uv = rnd(4, heads, kv_rank, dtype=dtype), rnd(heads, vdim, p8(kv_rank), dtype=dtype, scale=kv_rank ** -0.5)
    gate = rnd(T, p8(heads * vdim), dtype=dtype)
    out, gout = torch.zeros(T, p8(heads * vdim), dtype=dtype), torch.zeros(T, p8(heads * vdim), dtype=dtype, device=DEV)
    for g in (None, gate):
        ref.latent_values(o, rows, uv, heads, vdim, kv_rank, g, out)
        hops.latent_values(o.to(DEV), rows.to(DEV), uv.to(DEV), heads, vdim, kv_rank, None if g is None else g.to(DEV), gout)
        torch.testing.assert_close(gout.cpu(), out, **tol(dtype))


@pytest.mark.parametrize("kernel,dtype", [("simt", torch.float32), ("simt", torch.bfloat16), ("tc", torch.bfloat16)])
@pytest.mark.parametrize("heads,kv_rank,rot,page", [(3, 40, 16, 8), (16, 128, 32, 64), (20, 200, 24, 32), (40, 512, 64, 128),
                                                    (12, 512, 64, 32), (32, 448, 40, 64),
                                                    (5, 64, 64, 128)])
def test_latent_attention(kernel, dtype, heads, kv_rank, rot, page):
    lens = [1, 7, page, page + 1, 127, 128, 129, 400, 1500]
    row = hops.latent_row(kv_rank, rot)
    cache, bt = paged(lens, page, row, dtype)
    n = len(lens)
    qa = rnd(n, heads, row, dtype=dtype)
    scale = 1.5 * row ** -0.5
    # one key stands out for the last row: it sits on the first slot of a page, far back
    far = 2 * page if 2 * page < 1500 else 0
    flat = cache[bt[-1, far // page].long(), far % page]
    flat[:] = (qa[-1, 0].float() * 0.9).to(dtype)
    tok_seq, tok_kv = i32(range(n)), i32(lens)
    want = ref.latent_attention(qa, cache, tok_seq, tok_kv, bt, kv_rank, scale)
    out = torch.empty(n, heads, kv_rank, dtype=dtype, device=DEV)
    for max_len in (max(lens), 100 * max(lens)):         # the second asks for more splits than there are tiles
        hops.latent_attention(qa.to(DEV), cache.to(DEV), tok_seq.to(DEV), tok_kv.to(DEV), n, bt.to(DEV), kv_rank, scale,
                              out, max_len, kernel=kernel)
        torch.testing.assert_close(out.float().cpu(), want.float(), **tol(dtype))


@pytest.mark.parametrize("heads,dim,rot,vdim", [(3, 40, 16, 24), (2, 64, 32, 64), (4, 128, 64, 128), (2, 72, 8, 104),
                                                (2, 136, 32, 64)])
@pytest.mark.parametrize("q_lens,kv_lens", [([300], [300]), ([17, 128, 64], [40, 1000, 64]), ([2, 130], [130, 131])])
def test_latent_prefill(heads, dim, rot, vdim, q_lens, kv_lens):
    T, rows = sum(q_lens), sum(kv_lens)
    q, kv = rnd(T, heads * (dim + rot), dtype=torch.bfloat16), rnd(rows, heads * (dim + vdim), dtype=torch.bfloat16)
    lat = rnd(rows, 16 + rot, dtype=torch.bfloat16)
    gate = rnd(T, heads * vdim, dtype=torch.bfloat16)
    scale = 2.0 * (dim + rot) ** -0.5
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    begin = [sum(kv_lens[:b]) for b in range(len(kv_lens))]
    tiles = [(b, q0) for b, n in enumerate(q_lens) for q0 in range(0, n, 128)]
    want = torch.zeros(T, heads * vdim)
    for b, (n, m) in enumerate(zip(q_lens, kv_lens)):
        k = torch.cat([kv[begin[b]:begin[b] + m, :heads * dim].float().view(m, heads, dim),
                       lat[begin[b]:begin[b] + m, None, 16:].float().expand(m, heads, rot)], -1)
        v = kv[begin[b]:begin[b] + m, heads * dim:].float().view(m, heads, vdim)
        s = torch.einsum("qhd,khd->hqk", q[cu[b]:cu[b + 1]].float().view(n, heads, dim + rot), k) * scale
        s = s.masked_fill(torch.arange(m)[None] > torch.arange(m - n, m)[:, None], -math.inf)
        want[cu[b]:cu[b + 1]] = torch.einsum("hqk,khd->qhd", s.softmax(-1), v).reshape(n, -1)
    out = torch.zeros(T, heads * vdim, dtype=torch.bfloat16, device=DEV)
    g = lambda t: i32(t).to(DEV)
    for gt in (None, gate):
        hops.latent_prefill(q.to(DEV), kv.to(DEV), lat.to(DEV), 16, rows, g(begin), out, None if gt is None else gt.to(DEV),
                            g(cu), g(kv_lens), g([b for b, _ in tiles]), g([q0 for _, q0 in tiles]), len(tiles), heads, dim,
                            rot, vdim, scale)
        w = want if gt is None else want * torch.sigmoid(gate.float())
        torch.testing.assert_close(out.float().cpu(), w, atol=2e-2, rtol=2e-2)


def test_latent_gather():
    lens, page, row = [5, 130, 64, 33], 32, 24
    cache, bt = paged(lens, page, row, torch.bfloat16)
    seqs = [3, 1]
    cu = [0, 33, 163]
    out = torch.zeros(163, row, dtype=torch.bfloat16, device=DEV)
    hops.latent_gather(cache.to(DEV), i32(seqs).to(DEV), i32(cu).to(DEV), 130, bt.to(DEV), out)
    want = torch.cat([cache[bt[s].long()].reshape(-1, row)[: lens[s]] for s in seqs])
    assert torch.equal(out.cpu(), want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(40, 4), (37, 3), (64, 2), (24, 1), (300, 8)])
@pytest.mark.parametrize("q_lens,kv_lens", [([1, 1, 1], [1, 5, 2]), ([2, 1, 20, 9], [2, 4, 21, 9])])
def test_causal_conv(dtype, channels, taps, q_lens, kv_lens):
    T, B = sum(q_lens), len(q_lens)
    x, w, b = rnd(T, channels, dtype=dtype), rnd(taps, channels, dtype=dtype), rnd(channels, dtype=dtype)
    state = rnd(B + 2, taps - 1, channels, dtype=dtype)
    slots = torch.randperm(B + 2)[:B].int()
    cu = i32([sum(q_lens[:i]) for i in range(B + 1)])
    row_seq = i32([i for i, n in enumerate(q_lens) for _ in range(n)])
    out, gout, gs = torch.zeros(T, channels, dtype=dtype), torch.zeros(T, channels, dtype=dtype, device=DEV), state.to(DEV)
    ref.causal_conv(x, w, b, state, out, cu, i32(kv_lens), slots)
    hops.causal_conv(x.to(DEV), w.to(DEV), b.to(DEV), gs, gout, row_seq.to(DEV), cu.to(DEV), i32(kv_lens).to(DEV),
                     slots.to(DEV), max(q_lens) == 1)
    torch.testing.assert_close(gout.cpu(), out, **tol(dtype))
    assert torch.equal(gs.cpu(), state)


@pytest.mark.parametrize("form,dtype", [("scan", torch.float32), ("scan", torch.bfloat16), ("chunk", torch.bfloat16),
                                        ("chunk64", torch.bfloat16)])
@pytest.mark.parametrize("heads,vdim,N,groups", [(4, 40, 48, 2), (6, 64, 128, 1), (3, 72, 16, 3), (2, 24, 200, 1), (8, 8, 64, 8)])
def test_ssd(form, dtype, heads, vdim, N, groups):
    q_lens, kv_lens = [70, 1, 400, 64, 3, 128], [70, 9, 401, 500, 3, 129]
    T, B, inner = sum(q_lens), len(q_lens), heads * vdim
    xbc = rnd(T, inner + 2 * groups * N, dtype=dtype, scale=0.5)
    dt, bias = rnd(T, heads, dtype=dtype), rnd(heads, dtype=dtype, scale=0.5)
    A, D = (torch.rand(heads) * 2).to(dtype), rnd(heads, dtype=dtype)
    # a strong decay inside a chunk: what follows it is made of small differences of large running sums
    dt[20] += 40.0
    A[0] = 2.5
    state = rnd(B + 1, heads, vdim, N)
    slots = torch.randperm(B + 1)[:B].int()
    cu = i32([sum(q_lens[:i]) for i in range(B + 1)])
    y, gy, gs = torch.zeros(T, inner, dtype=dtype), torch.zeros(T, inner, dtype=dtype, device=DEV), state.to(DEV)
    seqs = i32(range(B))
    ref.ssd_scan(xbc, dt, bias, A, D, state, y, seqs, cu, i32(kv_lens), slots, groups)
    fn = {"scan": hops.ssd_scan, "chunk": hops.ssd_chunk, "chunk64": functools.partial(hops.ssd_chunk, form=1)}[form]
    fn(xbc.to(DEV), dt.to(DEV), bias.to(DEV), A.to(DEV), D.to(DEV), gs, gy, seqs.to(DEV), cu.to(DEV), i32(kv_lens).to(DEV),
       slots.to(DEV), groups)
    # the state is fp32 in every form: what the two-term products of the chunked form leave is far below bf16
    torch.testing.assert_close(gs.cpu(), state, atol=2e-4, rtol=2e-4)
    torch.testing.assert_close(gy.cpu(), y, **tol(dtype))

"""Giforax (``models/giforax.py``) beside the framework's closest models at equal size: throughput of prefill and decode,
and every kernel against its roofline and beside the like kernel's distance.

* ``throughput``: four layers (minGRU, attention, attention on the keys and values of the one before it, minGRU, each with a
  mixture of experts) and a Mixtral layout of the same width, heads and parameters, random weights and token ids, as in
  ``hybrid_bench.py``.
* ``kernels``: as there; the like kernels are those of the Mixtral layout (attention, router, grouped products, norms), of
  Netezen's routed layer and of Sidisun's recurrence.

``python bench.py --workload giforax`` runs both and prints one JSON line; ``python artifact/giforax_bench.py`` prints
tables.
"""
from __future__ import annotations

import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

from artifact.hybrid_bench import Timer, _i, _r, print_tables, throughput, with_ratios  # noqa: E402
from artifact.kebopel_bench import _Meta  # noqa: E402
from artifact.netezen_bench import visible  # noqa: E402

# width: heads, kv heads, recurrent channels, experts' feed-forward, shared one's
SIZES = {2048: (16, 4, 2048, 1024, 2048), 4096: (32, 8, 4096, 2048, 4096)}
EXPERTS, TOP = 16, 4                                     # (the Mixtral layout: 8 experts of twice the size, 2 per token)
D = 128
CHUNK = 4096
CLAMPED = ("clamped", 7.0, 1.702)


def models(width: int):
    from tokenweave_b200.config import ModelConfig, _giforax
    heads, kv, gru, ff, shared = SIZES[width]
    cfg = _giforax(32768, width, 4, (heads, kv, D, D, 64), gru, (EXPERTS, TOP, ff, 7.0), (shared, 7.0), CHUNK)
    giforax = ModelConfig.from_hf_dict(cfg, name=f"giforax-{width}")
    giforax.max_model_len = 16384
    # parameters: the shared experts as experts of the Mixtral layout
    inter = 3 * width * (EXPERTS * ff + shared) // (3 * width * 8) // 64 * 64
    mixtral = ModelConfig(name=f"mixtral-{width}", architecture="mixtral", num_q_heads=heads, num_kv_heads=kv, head_dim=D,
                          intermediate_size=inter, num_experts=8, num_experts_per_tok=2, hidden_size=width, num_layers=4,
                          vocab_size=32768, rms_norm_eps=1e-5, max_model_len=16384)
    return giforax, mixtral


def visible_in_chunks(T: int, chunk: int) -> int:
    """(query, key) pairs that a prompt of T tokens looks at."""
    return sum(i % chunk + 1 for i in range(T))


def kernels(width: int, T: int = 8192, batch: int = 128, context: int = 2048) -> list[dict]:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    from tokenweave_b200.ops import reference
    heads, hkv, gru, ff, shared = SIZES[width]
    t = Timer()
    cs, cs64 = (reference.build_cos_sin_cache(n, 16384, 500000.0, None, "cuda") for n in (D, 64))
    page, nb = 128, max(T // 128, batch * context // 128) + 8
    qkv_n = (heads + 2 * hkv) * D
    for m, tag in ((T, "prefill"), (batch, "decode")):
        single = tag == "decode"
        cu, kvl = (_i(range(m + 1)), _i([context] * m)) if single else (_i([0, m]), _i([m]))
        seqs = _i(range(m)) if single else _i([0])
        pos, slots = _i(range(m)), _i(range(128, 128 + m))
        meta = _Meta(positions=pos, slot_mapping=slots, cu_q=cu, kv_lens=kvl, num_seqs=seqs.shape[0], all_single=single, extra={})
        # norms, sums, averages, embedding
        w, b, y, res, xa = _r(width), _r(width), _r(m, width), _r(m, width), _r(m, width)
        x, results, norm = torch.randn(m, width, device="cuda"), torch.randn(33, m, width, device="cuda"), (w, b)
        t(f"add_rmsnorm [{tag}]", "", lambda: ops.add_rmsnorm_(y, res, w, 1e-5), m * width * 8)
        t(f"sandwich_step [{tag}]", f"add_rmsnorm [{tag}]",
          lambda: hops.sandwich_step(y, x, norm, norm, 1e-5, xa), m * width * 12)
        for past in (1, 4, 32):
            coef = torch.rand(past + 1, device="cuda")
            t(f"sandwich_step, average of {past + 1} [{tag}]", f"add_rmsnorm [{tag}]",
              lambda: hops.sandwich_step(y, x, norm, norm, 1e-5, xa, coef, results), m * width * (16 + 4 * past))
        t(f"sandwich_step, average of 5, last [{tag}]", f"add_rmsnorm [{tag}]",
          lambda: hops.sandwich_step(y, x, norm, norm, 1e-5, xa, coef[:5].contiguous(), results, True), m * width * (8 + 4 * 4))
        table = _r(32768, width)
        ids = torch.randint(0, 32768, (m,), dtype=torch.int32, device="cuda")
        t(f"embed_sandwich [{tag}]", f"embedding [{tag}]",
          lambda: hops.embed_sandwich(ids, table, 0.5, x, results[0], norm, 1e-5, xa), m * width * 12)
        t(f"embedding [{tag}]", "", lambda: ops.embedding(ids, table, out=y), m * width * 4)
        del table, x, results
        # between the projections and the attentions
        p, q = _r(m, qkv_n), _r(m, heads * D)
        kc, vc = (torch.zeros(m // page + 4, page, hkv, D, dtype=torch.bfloat16, device="cuda") for _ in range(2))
        wq = _r(D)
        t(f"rope_kv_write (head norm) [{tag}]", "",
          lambda: ops.rope_kv_write_(p, pos, slots, cs, kc, vc, heads, hkv, D, qk_norm=(wq, wq, 1e-5)), m * qkv_n * 4)
        prep = lambda g, k, v: hops.qkv_prep(p, heads, g, D, D, q, k, v, meta, None, None, "unit", None, None, 1e-5, 0.0, 1, cs64)
        t(f"qkv_prep (unit norm, rotation) [{tag}]", f"rope_kv_write (head norm) [{tag}]", lambda: prep(hkv, kc, vc), m * qkv_n * 4)
        t(f"qkv_prep, queries alone [{tag}]", f"rope_kv_write (head norm) [{tag}]", lambda: prep(0, None, None),
          m * heads * D * 4)
        del p, q, kc, vc
        # recurrence
        p, st, out = _r(m, 3 * gru), torch.randn(seqs.shape[0], gru, device="cuda"), _r(m, gru)
        bz, bx = torch.randn(gru, device="cuda") - 3.0, torch.randn(gru, device="cuda")
        run = lambda chunked: hops.min_gru(p, bz, bx, st, out, seqs, cu, kvl, seqs, chunked)
        # the like kernels: Mamba-2 with as many channels
        mh, chan = gru // 64, gru + 256
        xbc, dt, A, ys = _r(m, chan), _r(m, mh), _r(mh, scale=0.1), _r(m, gru)
        ss = torch.randn(seqs.shape[0], mh, 64, 128, device="cuda")
        state = seqs.shape[0] * mh * 64 * 128 * 8
        if single:
            t("ssd_scan [decode]", "", lambda: hops.ssd_scan(xbc, dt, A, A, A, ss, ys, seqs, cu, kvl, seqs, 1),
              m * (chan + gru) * 2 + state)
            t("min_gru [decode]", "add_rmsnorm [decode]", lambda: run(False), m * gru * 16)
        else:
            t("ssd_chunk [prefill]", "", lambda: hops.ssd_chunk(xbc, dt, A, A, A, ss, ys, seqs, cu, kvl, seqs, 1),
              m * (chan + gru) * 2 + state, 2.0 * m * (mh * 64 * 64 / 2 + 2 * mh * 128 * 64))
            t("min_gru [prefill]", "ssd_chunk [prefill]", lambda: run(True), m * gru * 8 + gru * 8)
            z = _r(gru)
            t("gated_group_norm [prefill]", "", lambda: hops.gated_group_norm(ys, out, z, 1, 1e-5, out), m * gru * 6)
            t("min_gru [prefill], beside a row kernel", "gated_group_norm [prefill]", lambda: run(True), m * gru * 8 + gru * 8)
        del p, xbc, ys, ss, out
        _experts(t, m, tag, width, ff, shared)
        for name, n, k, like in (("mixtral qkv", qkv_n, width, ""), ("in_proj (attention)", qkv_n + heads, width, "mixtral qkv"),
                                 ("in_proj (queries and gate)", heads * D + heads, width, "mixtral qkv"),
                                 ("in_proj (recurrence)", 3 * gru, width, "mixtral qkv"),
                                 ("out_proj", width, heads * D, "mixtral qkv")):
            a, c = _r(m, k), _r(n, k, scale=0.02)
            o = torch.empty(m, n, dtype=torch.bfloat16, device="cuda")
            t(f"gemm {name} [{tag}]", like and f"gemm {like} [{tag}]", lambda: ops.gemm(a, c, out=o), (m * k + n * k + m * n) * 2,
              2.0 * m * n * k)
        del a, c, o
    _attention(t, heads, hkv, T, batch, context, page, nb)
    return t.rows


def _experts(t, m, tag, width, ff, shared) -> None:
    from tokenweave_b200 import ops
    from tokenweave_b200.layers.moe import FusedMoE, expert_index, max_expert_rows, run_experts
    from tokenweave_b200.ops import hybrid as hops
    x, out = _r(m, width), _r(m, width)
    router = _r(EXPERTS, width, scale=width ** -0.5)
    nbytes, flops = (m * width + EXPERTS * width) * 2, 2.0 * m * EXPERTS * width
    t(f"moe_router (16 experts, top 4) [{tag}]", "", lambda: ops.moe_router(x, router, TOP), nbytes, flops)
    route = lambda: ops.moe_route(x, router, EXPERTS, TOP, None, 0.0, "sigmoid", False)
    t(f"moe_route (sigmoid scores) [{tag}]", f"moe_router (16 experts, top 4) [{tag}]", route, nbytes, flops)
    weights, ids, _ = route()
    used = len(set(ids.flatten().tolist()))
    ws, rows = expert_index(m, TOP, EXPERTS, "cuda"), max_expert_rows(m, TOP, EXPERTS)
    tile = 256 if m * TOP >= 512 * EXPERTS else 128
    n_rows = (m * TOP + EXPERTS * (tile - 1) + tile - 1) // tile * tile
    te = ws["tile_expert"][:n_rows // tile]
    a, mid, y = _r(rows, width), _r(rows, ff), _r(rows, width)
    ops.moe_align(ids, EXPERTS, tile, ws["offsets"], ws["cursor"], te, ws["meta"])
    pairs = m * TOP
    ops.moe_scatter(x, ids, weights, ws["offsets"], ws["cursor"], a, ws["row_scale"], ws["sorted_pos"], EXPERTS)
    sy = _r(m, width)
    t(f"moe_combine [{tag}]", "", lambda: ops.moe_combine(y, ws["sorted_pos"], out, TOP), (pairs + m) * width * 2)
    t(f"moe_combine + shared, no gate [{tag}]", f"moe_combine [{tag}]",
      lambda: ops.moe_combine(y, ws["sorted_pos"], out, TOP, sy), (pairs + 2 * m) * width * 2)
    w13, w2 = _r(EXPERTS * 2 * ff, width, scale=0.02), _r(EXPERTS * width, ff, scale=0.02)
    groups = dict(tile_expert=te, num_m_tiles=ws["meta"][:1], tile_rows=tile)
    silu = f"gemm experts gate_up + silu [{tag}]"
    for act, scale, name, like in (("silu", None, "experts gate_up + silu", ""),
                                   (CLAMPED, ws["row_scale"], "experts gate_up + clamped, weighted input", silu)):
        t(f"gemm {name} [{tag}]", like, lambda: ops.gemm(a[:n_rows], w13, out=mid[:n_rows], swiglu=True, act=act, in_scale=scale,
                                                         n_per_expert=2 * ff, **groups),
          (pairs * (width + ff) + used * 2 * ff * width) * 2, 4.0 * pairs * ff * width)
    t(f"gemm experts down [{tag}]", silu, lambda: ops.gemm(mid[:n_rows], w2, out=y[:n_rows], n_per_expert=width, **groups),
      (pairs * (width + ff) + used * ff * width) * 2, 2.0 * pairs * ff * width)
    # the whole layer beside the Mixtral layout of equal size (8 experts of twice the size, 2 per token)
    moe = FusedMoE(8, 2, width, 2 * ff, dtype=torch.bfloat16, device="cuda")
    for par in (moe.gate, moe.w13, moe.w2):
        par.data.normal_(0.0, 0.02)
    layer_bytes, layer_flops = (2 * m * width + EXPERTS * 3 * ff * width) * 2, 6.0 * pairs * ff * width
    t(f"mixtral experts (whole layer) [{tag}]", "", lambda: moe(x, out=out), layer_bytes, layer_flops)
    del moe

    def layer():
        w_, i_, _ = route()
        run_experts(x, w_, i_, w13.view(EXPERTS, 2 * ff, width), w2.view(EXPERTS, width, ff),
                    dict(ws, a_sorted=a, act=mid, y=y), out, CLAMPED, sy, None, weigh_input=True)
    t(f"routed experts (whole layer) [{tag}]", f"mixtral experts (whole layer) [{tag}]", layer, layer_bytes, layer_flops)
    del w13, w2, a, mid, y
    su, sa = _r(2 * shared, width, scale=0.02), _r(m, shared)
    for act, name, like in (("silu", "shared gate_up + silu", ""), (CLAMPED, "shared gate_up + clamped", f"gemm shared gate_up + silu [{tag}]")):
        t(f"gemm {name} [{tag}]", like, lambda: hops.gated_product(x, su, act, sa, None),
          (m * width + 2 * shared * width + m * shared) * 2, 4.0 * m * shared * width)


def _attention(t, heads, hkv, T, batch, context, page, nb) -> None:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    tiles, none, scale = T // 128, _i([]), D ** -0.5
    cu, kvl, ts = _i([0, T]), _i([T]), _i([0] * tiles)
    tq, bt = _i(list(reversed(range(0, T, 128)))), _i(range(1, T // page + 1)).view(1, -1)
    kc, vc = _r(nb, page, hkv, D), _r(nb, page, hkv, D)
    bias, pg = torch.full((heads,), -3.0, device="cuda"), _r(T, heads)
    meta = _Meta(num_tiles=tiles, num_single=0, cu_q=cu, kv_lens=kvl, block_table=bt, tile_seq=ts, tile_q0=tq, tok_row=none,
                 tok_seq=none, tok_kvlen=none, max_kv_len=T)
    q, o = _r(T, heads * D), _r(T, heads * D)
    nbytes, per_pair = (2 * q.numel() + 2 * T * hkv * D) * 2, 4.0 * heads * D
    t("attn_prefill", "", lambda: ops.attn_prefill(q, kc, vc, o, cu, kvl, bt, ts, tq, tiles, heads, hkv, D, scale), nbytes,
      per_pair * visible(T, T))
    t("grouped attention [prefill]", "attn_prefill",
      lambda: hops.grouped_attention(q, kc, vc, o, meta, heads, hkv, scale, None, False, 1.0), nbytes, per_pair * visible(T, T))
    sigmoid = lambda chunk: hops.grouped_attention(q, kc, vc, o, meta, heads, hkv, scale, None, False, 1.0, key_bias=bias,
                                                   chunk=chunk, gate=pg[:q.shape[0]])
    for chunk in (T, 2048, 512, 128):
        like = "attn_prefill"
        if chunk < T:
            # a window of half the chunk's size looks at about as many pairs
            like = f"attn_prefill, window {chunk // 2}"
            t(like, "", lambda: ops.attn_prefill(q, kc, vc, o, cu, kvl, bt, ts, tq, tiles, heads, hkv, D, scale,
                                                 window=chunk // 2), nbytes, per_pair * visible(T, chunk // 2))
        t(f"sigmoid attention, chunk {chunk} [prefill]", like, lambda: sigmoid(chunk), nbytes,
          per_pair * visible_in_chunks(T, chunk))
    # decode
    n, per = batch, context // page
    btd, tok, lens = _i([[1 + b * per + j for j in range(per)] for b in range(n)]), _i(range(n)), _i([context] * n)
    meta = _Meta(num_tiles=0, num_single=n, block_table=btd, tok_row=tok, tok_seq=tok, tok_kvlen=lens, max_kv_len=context)
    q, o = _r(n, heads * D), _r(n, heads * D)
    moved = lambda keys: n * keys * hkv * D * 4 + 4 * q.numel()
    t("attn_decode", "", lambda: ops.attn_decode(q, kc, vc, o, tok, tok, lens, n, btd, heads, hkv, D, scale, context),
      moved(context))
    for chunk in (context, 512, 128):
        like = "attn_decode"
        if chunk < context:
            like = f"attn_decode, window {chunk}"
            t(like, "", lambda: ops.attn_decode(q, kc, vc, o, tok, tok, lens, n, btd, heads, hkv, D, scale, context, window=chunk),
              moved(chunk))
        t(f"sigmoid attention, chunk {chunk} [decode]", like, lambda: sigmoid(chunk), moved(chunk))


def run(sizes=None, steps: int = 20) -> dict:
    out = {}
    for width in sizes or SIZES:
        giforax, mixtral = models(width)
        out[str(width)] = {"giforax": throughput(giforax, steps=steps), "mixtral": throughput(mixtral, steps=steps),
                           "kernels": with_ratios(kernels(width))}
    return out


if __name__ == "__main__":
    print_tables(run(), ("giforax", "mixtral"))

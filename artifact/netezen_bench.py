"""Netezen (``models/netezen.py``) beside the framework's closest models at equal size: throughput of prefill and decode,
and every kernel against its roofline and beside the like kernel's distance.

* ``throughput``: four layers (latent attention with a dense feed-forward, then attention, latent attention and attention
  with mixtures of experts) and a Mixtral layout of the same width, heads and parameters, random weights and token ids, as
  in ``hybrid_bench.py``.
* ``kernels``: as there; the like kernels are those of the Mixtral layout (attention, router, grouped products, norms) and
  of Sidisun's latent attention.

``python bench.py --workload netezen`` runs both and prints one JSON line; ``python artifact/netezen_bench.py`` prints
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

# width: heads, kv heads, kv_rank, q_rank, dense feed-forward, experts' feed-forward, shared one's
SIZES = {2048: (16, 4, 512, 768, 8192, 1024, 2048), 4096: (32, 8, 512, 1536, 16384, 2048, 4096)}
EXPERTS, TOP = 16, 4                                     # (the Mixtral layout: 8 experts of twice the size, 2 per token)
D, DIM, ROT, VDIM = 128, 128, 64, 128                    # head sizes of the attention and of the latent attention
STREAMS = 4
WINDOWS = (2048, 4, 1024)                                # attention, kept first tokens, latent attention
CLAMPED = ("clamped", 7.0, 1.702)


def models(width: int):
    from tokenweave_b200.config import ModelConfig, _netezen
    heads, kv, R, Q, dense, ff, shared = SIZES[width]
    cfg = _netezen(32768, width, 4, STREAMS, (heads, kv, D, D, 64), (heads, DIM, ROT, VDIM, R, Q), dense,
                   (EXPERTS, TOP, ff, 7.0), (shared, 7.0), WINDOWS)
    netezen = ModelConfig.from_hf_dict(cfg, name=f"netezen-{width}")
    netezen.max_model_len = 16384
    # parameters: the dense layer and the shared experts as experts of the Mixtral layout
    total = 2 * dense * width + 3 * (3 * width * (EXPERTS * ff + shared))
    inter = total // (4 * 3 * width * 8) // 64 * 64
    mixtral = ModelConfig(name=f"mixtral-{width}", architecture="mixtral", num_q_heads=heads, num_kv_heads=kv, head_dim=D,
                          intermediate_size=inter, num_experts=8, num_experts_per_tok=2, hidden_size=width, num_layers=4,
                          vocab_size=32768, rms_norm_eps=1e-5, max_model_len=16384)
    return netezen, mixtral


def visible(T: int, window: int, keep: int = 0) -> int:
    """(query, key) pairs that a prompt of T tokens looks at."""
    return sum(min(i + 1, window) + min(max(0, i + 1 - window), keep) for i in range(T))


def kernels(width: int, T: int = 8192, batch: int = 128, context: int = 2048) -> list[dict]:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    from tokenweave_b200.ops import reference
    heads, hkv, R, Q, dense, ff, shared = SIZES[width]
    t = Timer()
    cs, cs64 = (reference.build_cos_sin_cache(n, 16384, 500000.0, None, "cuda") for n in (D, 64))
    page, nb = 128, max(T // 128, batch * context // 128) + 8
    qkv_n, row = (heads + 2 * hkv) * D, hops.latent_row(R, ROT)
    for m, tag in ((T, "prefill"), (batch, "decode")):
        pos, slots = _i(range(m)), _i(range(128, 128 + m))
        meta = _Meta(positions=pos, slot_mapping=slots, cu_q=_i([0, m]), kv_lens=_i([m]), num_seqs=1, all_single=False, extra={})
        # streams, norms, embedding
        w, y, res, xa = _r(width), _r(m, width), _r(m, width), _r(m, width)
        x = torch.randn(m, STREAMS, width, device="cuda")
        c = torch.rand(STREAMS, device="cuda")
        hc = {"in": c, "out": c, "mix": torch.eye(STREAMS, device="cuda")}
        t(f"streams_step [{tag}]", f"add_rmsnorm [{tag}]",
          lambda: hops.streams_step(y, x, hc, 0.5, c, w, 1.0, 1e-5, xa), m * width * (8 * STREAMS + 4))
        t(f"streams_step, last [{tag}]", f"add_rmsnorm [{tag}]",
          lambda: hops.streams_step(y, x, hc, 0.5, None, w, 1.0, 1e-5, xa), m * width * (4 * STREAMS + 4))
        t(f"add_rmsnorm [{tag}]", "", lambda: ops.add_rmsnorm_(y, res, w, 1e-5), m * width * 8)
        table = _r(32768, width)
        ids = torch.randint(0, 32768, (m,), dtype=torch.int32, device="cuda")
        t(f"embed_streams [{tag}]", f"embedding [{tag}]",
          lambda: hops.embed_streams(ids, table, x, c, w, 1.0, 1e-5, xa), m * width * 8)
        t(f"streams_step, first [{tag}]", f"add_rmsnorm [{tag}]",
          lambda: hops.streams_step(y, x, hc, 0.5, c, w, 1.0, 1e-5, xa, first=True), m * width * (4 * STREAMS + 8))
        t(f"embedding [{tag}]", "", lambda: ops.embedding(ids, table, out=y), m * width * 4)
        del table, x
        # between the projections and the attentions
        p, q = _r(m, qkv_n), _r(m, heads * D)
        kc, vc = (torch.zeros(m // page + 4, page, hkv, D, dtype=torch.bfloat16, device="cuda") for _ in range(2))
        t(f"qkv_prep (rotation) [{tag}]", f"rope_kv_write [{tag}]",
          lambda: hops.qkv_prep(p, heads, hkv, D, D, q, kc, vc, meta, None, None, None, None, None, 1e-5, 0.0, 1, cs64),
          m * qkv_n * 4)
        t(f"rope_kv_write [{tag}]", "", lambda: ops.rope_kv_write_(p, pos, slots, cs, kc, vc, heads, hkv, D),
          m * (2 * heads + 4 * hkv) * D * 2)
        kv8 = (R + ROT + 7) // 8 * 8
        pr, cq, wq, wkv = _r(m, Q + kv8), _r(m, Q), _r(Q), _r(R)
        cache = torch.zeros(nb, page, row, dtype=torch.bfloat16, device="cuda")
        t(f"latent_prep [{tag}]", f"rope_kv_write [{tag}]",
          lambda: hops.latent_prep(pr, 0, Q, wq, cq, Q, R, wkv, ROT, ROT, cs64, pos, slots, cache, 1e-5),
          m * (2 * Q + 2 * (R + ROT)) * 2)
        del p, q, pr, cache
        _experts(t, m, tag, width, ff, shared)
        # products with an activation, and those both models have
        a = _r(m, width)
        for act, name, like in ((None, "llama up (plain)", ""), ("relu2", "up + relu^2", f"gemm llama up (plain) [{tag}]")):
            b, o = _r(dense, width, scale=0.02), _r(m, dense)
            t(f"gemm {name} [{tag}]", like, lambda: hops.projection(a, b, None, (0, dense) if act else None, o, act or "silu"),
              (m * width + dense * width + m * dense) * 2, 2.0 * m * dense * width)
        for name, n, k, like in (("mixtral qkv", qkv_n, width, ""), ("in_proj (latent)", Q + kv8, width, "mixtral qkv"),
                                 ("uq_proj (latent)", heads * (DIM + ROT), Q, "mixtral qkv"),
                                 ("out_proj", width, heads * D, "mixtral qkv")):
            a, b = _r(m, k), _r(n, k, scale=0.02)
            o = torch.empty(m, n, dtype=torch.bfloat16, device="cuda")
            t(f"gemm {name} [{tag}]", like and f"gemm {like} [{tag}]", lambda: ops.gemm(a, b, out=o), (m * k + n * k + m * n) * 2,
              2.0 * m * n * k)
        del a, b, o
    _attention(t, heads, hkv, R, row, T, batch, context, page, nb, cs64)
    return t.rows


def _experts(t, m, tag, width, ff, shared) -> None:
    from tokenweave_b200 import ops
    from tokenweave_b200.layers.moe import FusedMoE, expert_index, max_expert_rows
    from tokenweave_b200.ops import hybrid as hops
    x, out = _r(m, width), _r(m, width)
    router = _r(EXPERTS + 1, width, scale=width ** -0.5)
    corr = torch.zeros(EXPERTS, device="cuda")
    nbytes, flops = (m * width + EXPERTS * width) * 2, 2.0 * m * EXPERTS * width
    t(f"moe_route (softmax, correction, gate) [{tag}]", f"moe_router (16 experts, top 4) [{tag}]",
      lambda: ops.moe_route(x, router, EXPERTS, TOP, corr, 1e-20), nbytes, flops)
    t(f"moe_router (16 experts, top 4) [{tag}]", "", lambda: ops.moe_router(x, router[:EXPERTS], TOP), nbytes, flops)
    weights, ids, gates = ops.moe_route(x, router, EXPERTS, TOP, corr, 1e-20)
    used = len(set(ids.flatten().tolist()))
    ws, rows = expert_index(m, TOP, EXPERTS, "cuda"), max_expert_rows(m, TOP, EXPERTS)
    tile = 256 if m * TOP >= 512 * EXPERTS else 128
    n_rows = (m * TOP + EXPERTS * (tile - 1) + tile - 1) // tile * tile
    te = ws["tile_expert"][:n_rows // tile]
    a, mid, y = _r(rows, width), _r(rows, ff), _r(rows, width)
    ops.moe_align(ids, EXPERTS, tile, ws["offsets"], ws["cursor"], te, ws["meta"])
    pairs = m * TOP

    def scatter():
        ws["cursor"].zero_()
        ops.moe_scatter(x, ids, weights, ws["offsets"], ws["cursor"], a, ws["row_scale"], ws["sorted_pos"], EXPERTS)
    t(f"moe_scatter (+ a memset) [{tag}]", "", scatter, (m + pairs) * width * 2)
    sy, gate = _r(m, width), gates[:, 0].contiguous()
    t(f"moe_combine + shared [{tag}]", f"moe_combine [{tag}]",
      lambda: ops.moe_combine(y, ws["sorted_pos"], out, TOP, sy, gate), (pairs + 2 * m) * width * 2)
    t(f"moe_combine [{tag}]", "", lambda: ops.moe_combine(y, ws["sorted_pos"], out, TOP), (pairs + m) * width * 2)
    w13, w2 = _r(EXPERTS * 2 * ff, width, scale=0.02), _r(EXPERTS * width, ff, scale=0.02)
    groups = dict(tile_expert=te, num_m_tiles=ws["meta"][:1], tile_rows=tile)
    for act, name, like in (("silu", "experts gate_up + silu", ""), (CLAMPED, "experts gate_up + clamped", f"gemm experts gate_up + silu [{tag}]")):
        t(f"gemm {name} [{tag}]", like, lambda: ops.gemm(a[:n_rows], w13, out=mid[:n_rows], swiglu=True, act=act,
                                                         n_per_expert=2 * ff, **groups),
          (pairs * (width + ff) + used * 2 * ff * width) * 2, 4.0 * pairs * ff * width)
    t(f"gemm experts down [{tag}]", f"gemm experts gate_up + silu [{tag}]",
      lambda: ops.gemm(mid[:n_rows], w2, out=y[:n_rows], row_scale=ws["row_scale"], n_per_expert=width, **groups),
      (pairs * (width + ff) + used * ff * width) * 2, 2.0 * pairs * ff * width)
    # the whole layer beside the Mixtral layer of equal size (8 experts of twice the size, 2 per token)
    moe = FusedMoE(8, 2, width, 2 * ff, dtype=torch.bfloat16, device="cuda")
    for par in (moe.gate, moe.w13, moe.w2):
        par.data.normal_(0.0, 0.02)
    layer_bytes, layer_flops = (2 * m * width + EXPERTS * 3 * ff * width) * 2, 6.0 * pairs * ff * width
    t(f"mixtral experts (whole layer) [{tag}]", "", lambda: moe(x, out=out), layer_bytes, layer_flops)
    del moe

    def layer():
        from tokenweave_b200.layers.moe import run_experts
        w_, i_, _ = ops.moe_route(x, router, EXPERTS, TOP, corr, 1e-20)
        run_experts(x, w_, i_, w13.view(EXPERTS, 2 * ff, width), w2.view(EXPERTS, width, ff),
                    dict(ws, a_sorted=a, act=mid, y=y), out, CLAMPED, sy, gate)
    t(f"routed experts (whole layer) [{tag}]", f"mixtral experts (whole layer) [{tag}]", layer, layer_bytes, layer_flops)
    del w13, w2, a, mid, y
    su, sa = _r(2 * shared, width, scale=0.02), _r(m, shared)
    for act, name, like in (("silu", "shared gate_up + silu", ""), (CLAMPED, "shared gate_up + clamped", f"gemm shared gate_up + silu [{tag}]")):
        t(f"gemm {name} [{tag}]", like, lambda: hops.gated_product(x, su, act, sa, None),
          (m * width + 2 * shared * width + m * shared) * 2, 4.0 * m * shared * width)


def _attention(t, heads, hkv, R, row, T, batch, context, page, nb, cs64) -> None:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    tiles, none = T // 128, _i([])
    cu, kvl, ts = _i([0, T]), _i([T]), _i([0] * tiles)
    tq, bt = _i(list(reversed(range(0, T, 128)))), _i(range(1, T // page + 1)).view(1, -1)
    # grouped attention: prefill
    scale = D ** -0.5
    kc, vc = _r(nb, page, hkv, D), _r(nb, page, hkv, D)
    meta = _Meta(num_tiles=tiles, num_single=0, cu_q=cu, kv_lens=kvl, block_table=bt, tile_seq=ts, tile_q0=tq, tok_row=none,
                 tok_seq=none, tok_kvlen=none, max_kv_len=T)
    q, o = _r(T, heads * D), _r(T, heads * D)
    nbytes = (2 * q.numel() + 2 * T * hkv * D) * 2
    for window in (2048, 512, 128):
        flops = 4.0 * heads * D * visible(T, window)
        t(f"attn_prefill, window {window}", "", lambda: ops.attn_prefill(q, kc, vc, o, cu, kvl, bt, ts, tq, tiles, heads, hkv, D,
                                                                         scale, window=window), nbytes, flops)
        t(f"windowed attention, {window} + 4 kept [prefill]", f"attn_prefill, window {window}",
          lambda: hops.grouped_attention(q, kc, vc, o, meta, heads, hkv, scale, None, False, 1.0, window=window, keep=4),
          nbytes, 4.0 * heads * D * visible(T, window, 4))
    # decode
    n, per = batch, context // page
    btd, tok, lens = _i([[1 + b * per + j for j in range(per)] for b in range(n)]), _i(range(n)), _i([context] * n)
    meta = _Meta(num_tiles=0, num_single=n, block_table=btd, tok_row=tok, tok_seq=tok, tok_kvlen=lens, max_kv_len=context)
    q, o = _r(n, heads * D), _r(n, heads * D)
    moved = lambda keys: n * keys * hkv * D * 4 + 4 * q.numel()
    t("attn_decode", "", lambda: ops.attn_decode(q, kc, vc, o, tok, tok, lens, n, btd, heads, hkv, D, scale, context),
      moved(context))
    for window in (2048, 512, 128):
        keys = min(window + 4, context)
        t(f"attn_decode, window {window}", "", lambda: ops.attn_decode(q, kc, vc, o, tok, tok, lens, n, btd, heads, hkv, D, scale,
                                                                       context, window=window), moved(min(window, context)))
        t(f"windowed attention, {window} + 4 kept [decode]", f"attn_decode, window {window}" if window < context else "attn_decode",
          lambda: hops.grouped_attention(q, kc, vc, o, meta, heads, hkv, scale, None, False, 1.0, window=window, keep=4),
          moved(keys))
    del q, o, kc, vc
    # latent attention: prefill
    scale, sink = (DIM + ROT) ** -0.5, torch.zeros(heads, device="cuda")
    q, kv, lat = _r(T, heads * (DIM + ROT)), _r(T, heads * (DIM + VDIM)), _r(T, row)
    out, begin = _r(T, heads * VDIM), _i([0])
    nbytes = (q.numel() + kv.numel() + out.numel()) * 2
    run = lambda window, s: hops.latent_prefill(q, kv, lat, R, T, begin, out, None, cu, kvl, ts, tq, tiles, heads, DIM, ROT, VDIM,
                                                scale, window, s)
    t("latent_prefill", "", lambda: run(0, None), nbytes, 2.0 * heads * visible(T, T) * (DIM + ROT + VDIM))
    for window in (T, 1024, 128):
        t(f"latent_prefill, window {window} + sink", "latent_prefill" if window >= 1024 else "attn_prefill, window 128",
          lambda: run(window, sink), nbytes, 2.0 * heads * visible(T, window) * (DIM + ROT + VDIM))
    pos = _i(range(T))
    t("rope_tail", "rope_kv_write [prefill]", lambda: hops.rope_tail_(q, heads, DIM + ROT, DIM, ROT, cs64, pos),
      T * heads * ROT * 4)
    cache = _r(nb, page, row)
    cc = _i([0, T])
    t("latent_gather", "", lambda: hops.latent_gather(cache, begin, cc, T, bt, lat, begin), T * row * 4)
    wkv, kvo = _r(heads * (DIM + VDIM), R, scale=0.04), torch.empty_like(kv)
    t("gemm ukv_proj (expand)", "gemm mixtral qkv [prefill]", lambda: ops.gemm(lat[:, :R], wkv, out=kvo),
      (T * R + wkv.numel() + kvo.numel()) * 2, 2.0 * T * R * heads * (DIM + VDIM))
    del q, kv, out, kvo
    # decode
    qa, o = _r(n, heads, row), _r(n, heads, R)
    moved = lambda keys: n * keys * row * 2 + qa.numel() * 2 + o.numel() * 2
    run = lambda window, s: hops.latent_attention(qa, cache, tok, lens, n, btd, R, scale, o, context, window=window, sink=s)
    t("latent_decode", "", lambda: run(0, None), moved(context))
    for window in (2048, 1024, 128):
        t(f"latent_decode, window {window} + sink", "latent_decode" if window >= 1024 else "attn_decode, window 128",
          lambda: run(window, sink), moved(window))
    q, ukt = _r(n, heads * (DIM + ROT)), _r(heads, R, DIM, scale=0.09)
    t("latent_absorb (head_gemm + latent_query)", "gemm mixtral qkv [decode]",
      lambda: hops.latent_absorb(q, tok, ukt, heads, DIM, ROT, ROT, R, cs64, lens, qa),
      (q.numel() + ukt.numel() + qa.numel()) * 2, 2.0 * n * heads * DIM * R)
    uv, at = _r(heads, VDIM, R, scale=0.04), _r(n, heads * VDIM)
    t("latent_values (head_gemm)", "gemm mixtral qkv [decode]",
      lambda: hops.latent_values(o, tok, uv, heads, VDIM, R, None, at), (o.numel() + uv.numel() + at.numel()) * 2,
      2.0 * n * heads * VDIM * R)


def run(sizes=None, steps: int = 20) -> dict:
    out = {}
    for width in sizes or SIZES:
        netezen, mixtral = models(width)
        out[str(width)] = {"netezen": throughput(netezen, steps=steps), "mixtral": throughput(mixtral, steps=steps),
                           "kernels": with_ratios(kernels(width))}
    return out


if __name__ == "__main__":
    print_tables(run(), ("netezen", "mixtral"))

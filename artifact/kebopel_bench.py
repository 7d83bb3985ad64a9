"""Kebopel (``models/kebopel.py``) beside the framework's closest models at equal size: throughput of prefill and decode,
and every kernel against its roofline and beside the like kernel's distance.

* ``throughput``: four layers (three pairs of biased and lightning attention, one convolved attention) and a Llama layout of
  the same width, heads and parameters, random weights and token ids, as in ``hybrid_bench.py``.
* ``kernels``: as there; the like kernels are those of the Llama layout (attention, projections, sums and norms) and of
  the Mamba-2 layers (recurrence, gated norm).

``python bench.py --workload kebopel`` runs both and prints one JSON line; ``python artifact/kebopel_bench.py`` prints
tables.
"""
from __future__ import annotations

import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

from artifact.hybrid_bench import Timer, _i, _r, print_tables, throughput, with_ratios  # noqa: E402

SIZES = {2048: (16, 4, 16, 7168), 4096: (32, 8, 32, 14336)}     # width: heads, kv heads, lightning heads, feed-forward
D = 128                                                        # every head size
TAPS = 4


def models(width: int):
    from tokenweave_b200.config import ModelConfig, _decays, _kebopel
    heads, kv, lh, ff = SIZES[width]
    cfg = _kebopel(32768, width, ff, 4, (heads, kv, D, D), (heads, kv, D, D), (lh, D, D), _decays(lh), None, 65536)
    kebopel = ModelConfig.from_hf_dict(cfg, name=f"kebopel-{width}")
    kebopel.max_model_len = 16384
    attn = width * (heads + 2 * kv) * D + heads * D * width
    extra = 3 * (width * 4 * lh * D + lh * D * width) // (4 * 3 * width) // 64 * 64      # the lightning sides' parameters
    llama = ModelConfig(name=f"llama-{width}", architecture="llama", num_q_heads=heads, num_kv_heads=kv, head_dim=D,
                        intermediate_size=ff + extra, hidden_size=width, num_layers=4, vocab_size=32768,
                        rms_norm_eps=1e-5, max_model_len=16384)
    assert abs(4 * (attn + 3 * width * (ff + extra)) / (4 * (attn + 3 * width * ff) + 15 * width * lh * D) - 1) < 0.02
    return kebopel, llama


class _Meta:
    """The fields of a step's metadata that the operators read."""

    def __init__(self, **kw):
        self.__dict__.update(kw)


def kernels(width: int, T: int = 8192, batch: int = 128, context: int = 2048) -> list[dict]:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    from tokenweave_b200.ops import reference
    heads, hkv, lh, ff = SIZES[width]
    t = Timer()
    cs = reference.build_cos_sin_cache(D, 16384, 500000.0, None, "cuda")
    page, nb = 128, max(T // 128, batch * context // 128) + 8
    qkv_n, inner = (heads + 2 * hkv) * D, lh * D
    for m, tag in ((T, "prefill"), (batch, "decode")):
        single = tag == "decode"
        cu = _i(range(m + 1)) if single else _i([0, m])
        kvl = _i([context] * m) if single else _i([m])
        seqs = _i(range(m)) if single else _i([0])
        rs = _i(range(m)) if single else _i([0] * m)
        pos, slots = _i([context - 1] * m) if single else _i(range(m)), _i(range(128, 128 + m))
        meta = _Meta(positions=pos, slot_mapping=slots, cu_q=cu, kv_lens=kvl, num_seqs=seqs.shape[0], all_single=single,
                     extra={"row_seq": rs, "state_slots": seqs, "prev_token": seqs})
        # sums, norms, embedding
        w, x, res, xa = _r(width), _r(m, width), _r(m, width), _r(m, width)
        x32, first = torch.randn(m, width, device="cuda"), torch.randn(m, width, device="cuda")
        t(f"add_prenorm [{tag}]", f"add_rmsnorm [{tag}]", lambda: hops.add_prenorm_(x, x32, None, w, 1e-5, xa), m * width * 12)
        t(f"add_prenorm + first [{tag}]", f"add_rmsnorm [{tag}]", lambda: hops.add_prenorm_(x, x32, first, w, 1e-5, xa),
          m * width * 16)
        t(f"add_rmsnorm [{tag}]", "", lambda: ops.add_rmsnorm_(x, res, w, 1e-5), m * width * 8)
        table, pairs = _r(32768, width), _r(65537, width)
        ids = torch.randint(0, 32768, (m,), dtype=torch.int32, device="cuda")
        spec = dict(buckets=65536, mul_prev=8191, mul_cur=31)
        t(f"embed_norm [{tag}]", f"embedding [{tag}]",
          lambda: hops.embed_norm(ids, table, pairs, spec, meta, x32, None, w, 1e-5, xa), m * width * 10)
        t(f"embedding [{tag}]", "", lambda: ops.embedding(ids, table, out=x), m * width * 4)
        del table, pairs
        # between projection and attention
        p, q = _r(m, qkv_n), _r(m, heads * D)
        kc, vc = (torch.zeros(m // page + 4, page, hkv, D, dtype=torch.bfloat16, device="cuda") for _ in range(2))
        cw, cst = _r(TAPS, qkv_n), _r(batch, TAPS - 1, qkv_n)
        wq, wk, whq, whk = _r(D), _r(D), _r(heads * D), _r(hkv * D)
        t(f"qkv_prep (convolution, head norm) [{tag}]", f"rope_kv_write (head norm) [{tag}]",
          lambda: hops.qkv_prep(p, heads, hkv, D, D, q, kc, vc, meta, cw, cst, "head", wq, wk, 1e-5, 0.1, 8192),
          m * qkv_n * 4 + (m * 2 * (TAPS - 1) * qkv_n * 2 if single else 0))
        t(f"qkv_prep (whole norm) [{tag}]", f"rope_kv_write (head norm) [{tag}]",
          lambda: hops.qkv_prep(p, heads, hkv, D, D, q, kc, vc, meta, None, None, "whole", whq, whk, 1e-5, 0.0, 1),
          m * qkv_n * 4)
        t(f"rope_kv_write (head norm) [{tag}]", "",
          lambda: ops.rope_kv_write_(p, pos, slots, cs, kc, vc, heads, hkv, D, qk_norm=(wq, wk, 1e-5)), m * qkv_n * 4)
        # recurrence, its norm and gate
        n_in = 4 * inner
        pr, ys, out, wn, decay = _r(m, n_in, scale=0.3), _r(m, inner), _r(m, inner), _r(inner), torch.rand(lh, device="cuda")
        st = torch.randn(seqs.shape[0], lh, D, D, device="cuda")
        t(f"norm_gate [{tag}]", f"gated_group_norm [{tag}]",
          lambda: hops.norm_gate(ys, pr[:, 3 * inner:], wn, inner, 1e-5, 0.7, out), m * inner * 6)
        t(f"gated_group_norm [{tag}]", "", lambda: hops.gated_group_norm(ys, pr[:, 3 * inner:], wn, 1, 1e-5, out), m * inner * 6)
        dt, bias, A, skip = _r(m, lh), _r(lh, scale=0.1), _r(lh, scale=0.1), _r(lh)
        if single:
            nbytes = m * (lh * D * D * 8 + 4 * inner * 2)
            t("decay_scan [decode]", "ssd_scan [decode]", lambda: hops.decay_scan(pr, decay, st, ys, seqs, cu, kvl, seqs), nbytes)
            t("ssd_scan [decode]", "", lambda: hops.ssd_scan(pr, dt, bias, A, skip, st, ys, seqs, cu, kvl, seqs, lh), nbytes)
        else:
            nbytes, flops = m * 4 * inner * 2 + lh * D * D * 8, 2.0 * m * lh * (64 * D / 2 + 64 * D / 2 + 2 * D * D)
            t("decay_chunk [prefill]", "ssd_chunk [prefill]", lambda: hops.decay_chunk(pr, decay, st, ys, seqs, cu, kvl, seqs),
              nbytes, flops)
            t("ssd_chunk [prefill]", "", lambda: hops.ssd_chunk(pr, dt, bias, A, skip, st, ys, seqs, cu, kvl, seqs, lh), nbytes,
              flops)
        del p, q, pr, ys, out, st
        # matrix products
        x = _r(m, width)
        for name, n, silu in (("in_proj + silu (pair)", qkv_n + n_in, (qkv_n, qkv_n + 3 * inner)), ("in_proj (attention)", qkv_n, None)):
            b, c, bias_v = _r(n, width, scale=0.02), _r(m, n), None if silu else _r(n)
            t(f"gemm {name} [{tag}]", f"gemm llama qkv [{tag}]", lambda: hops.projection(x, b, bias_v, silu, c),
              (m * width + n * width + m * n) * 2, 2.0 * m * n * width)
        b, c = _r(qkv_n, width, scale=0.02), _r(m, qkv_n)
        t(f"gemm llama qkv [{tag}]", "", lambda: ops.gemm(x, b, out=c), (m * width + qkv_n * width + m * qkv_n) * 2,
          2.0 * m * qkv_n * width)
        b, c = _r(2 * ff, width, scale=0.02), _r(m, ff)
        for act, name, like in (("gelu_tanh", "gate_up + gelu", f"gemm llama gate_up + silu [{tag}]"), ("silu", "llama gate_up + silu", "")):
            t(f"gemm {name} [{tag}]", like, lambda: hops.gated_product(x, b, act, c, None), (m * width + 2 * ff * width + m * ff) * 2,
              4.0 * m * ff * width)
        for name, k, like in (("out_proj (pair)", heads * D + inner + ff, f"gemm llama down [{tag}]"),
                              ("out_proj (attention)", heads * D + ff, f"gemm llama down [{tag}]"), ("llama down", ff, "")):
            a, b, c = _r(m, k), _r(width, k, scale=0.02), _r(m, width)
            t(f"gemm {name} [{tag}]", like, lambda: ops.gemm(a, b, out=c), (m * k + width * k + m * width) * 2, 2.0 * m * width * k)
        del a, b, c, x
    _attention(t, heads, hkv, T, batch, context, page, nb)
    return t.rows


def _attention(t, heads, hkv, T, batch, context, page, nb) -> None:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    scale, tiles = D ** -0.5, T // 128
    slopes = torch.exp2(-8.0 * torch.arange(1, heads + 1, device="cuda") / heads)
    kc, vc = _r(nb, page, hkv, D), _r(nb, page, hkv, D)
    cu, kvl, ts = _i([0, T]), _i([T]), _i([0] * tiles)
    tq, bt = _i(list(reversed(range(0, T, 128)))), _i(range(1, T // page + 1)).view(1, -1)
    none = _i([])
    meta = _Meta(num_tiles=tiles, num_single=0, cu_q=cu, kv_lens=kvl, block_table=bt, tile_seq=ts, tile_q0=tq, tok_row=none,
                 tok_seq=none, tok_kvlen=none, max_kv_len=T)
    q, o = _r(T, heads * D), _r(T, heads * D)
    nbytes, flops = (2 * q.numel() + 2 * T * hkv * D) * 2, 2.0 * heads * T * T / 2 * 2 * D
    for name, sl, sink in (("grouped attention", None, False), ("grouped attention, bias + sink", slopes, True)):
        t(f"{name} [prefill]", "attn_prefill", lambda: hops.grouped_attention(q, kc, vc, o, meta, heads, hkv, scale, sl, sink, 0.7),
          nbytes, flops)
    t("attn_prefill", "", lambda: ops.attn_prefill(q, kc, vc, o, cu, kvl, bt, ts, tq, tiles, heads, hkv, D, scale), nbytes, flops)
    n, per = batch, context // page
    btd, tok, lens = _i([[1 + b * per + j for j in range(per)] for b in range(n)]), _i(range(n)), _i([context] * n)
    meta = _Meta(num_tiles=0, num_single=n, block_table=btd, tok_row=tok, tok_seq=tok, tok_kvlen=lens, max_kv_len=context)
    q, o = _r(n, heads * D), _r(n, heads * D)
    nbytes, flops = n * context * hkv * D * 4 + 4 * q.numel(), 2.0 * n * heads * context * 2 * D
    for name, sl, sink in (("grouped attention", None, False), ("grouped attention, bias + sink", slopes, True)):
        t(f"{name} [decode]", "attn_decode", lambda: hops.grouped_attention(q, kc, vc, o, meta, heads, hkv, scale, sl, sink, 0.7),
          nbytes, flops)
    t("attn_decode", "", lambda: ops.attn_decode(q, kc, vc, o, tok, tok, lens, n, btd, heads, hkv, D, scale, context), nbytes, flops)


def run(sizes=None, steps: int = 20) -> dict:
    out = {}
    for width in sizes or SIZES:
        kebopel, llama = models(width)
        out[str(width)] = {"kebopel": throughput(kebopel, steps=steps), "llama": throughput(llama, steps=steps),
                           "kernels": with_ratios(kernels(width))}
    return out


if __name__ == "__main__":
    print_tables(run(), ("kebopel", "llama"))

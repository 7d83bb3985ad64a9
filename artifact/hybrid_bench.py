"""Hybrid decoder (latent attention + Mamba-2 layers, ``models/sidisun.py``) beside the framework's closest uniform model
(the Llama layout) at equal size: throughput of prefill and decode, and every kernel against its roofline.

* ``throughput``: four layers (three Mamba-2, one latent attention; the Llama model has four of its own with the same
  width, head count and feed-forward parameters), random weights and token ids, through ``LLM.generate``; device time of
  the steps from CUDA events around them, decode steps replayed from CUDA graphs in both models.
* ``kernels``: each launch alone, L2 flushed between iterations, median of the iterations; roofline time = the larger of
  bytes / measured copy bandwidth and FLOPs / measured bf16 rate (``MEASURED_PEAKS.json``).

``python bench.py --workload hybrid`` runs both and prints one JSON line; ``python artifact/hybrid_bench.py`` prints
tables.
"""
from __future__ import annotations

import json
import os
import statistics
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

SIZES = {          # width: (heads, kv_rank, q_rank, feed-forward of the hybrid model, Mamba-2 heads, groups)
    2048: (16, 512, 768, 8192, 64, 1),
    4096: (32, 512, 1536, 16384, 128, 8),
}
DIM, ROT, VDIM, P, N, TAPS = 128, 64, 128, 64, 128, 4


def peaks() -> tuple[float, float]:
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    return 6.65e12, 1.59e15


def models(width: int):
    from tokenweave_b200.config import ModelConfig, _latent_layer, _mamba2_layer
    heads, kv, q, ff, mh, groups = SIZES[width]
    layers = [_mamba2_layer(mh, P, N, groups, ff, conv=TAPS, norm_groups=groups) for _ in range(3)]
    layers.append(_latent_layer(heads, DIM, ROT, VDIM, kv, q, ff, base=500000.0))
    common = dict(hidden_size=width, num_layers=4, vocab_size=32768, rms_norm_eps=1e-5, max_model_len=16384)
    hybrid = ModelConfig(name=f"sidisun-{width}", architecture="sidisun", num_q_heads=heads, num_kv_heads=1,
                         head_dim=DIM + ROT, intermediate_size=ff, layers=layers, **common)
    llama = ModelConfig(name=f"llama-{width}", architecture="llama", num_q_heads=heads, num_kv_heads=heads // 4,
                        head_dim=128, intermediate_size=ff * 2 // 3 // 64 * 64, **common)
    return hybrid, llama


# ---- throughput ------------------------------------------------------------------------------------------------------
def throughput(cfg, prompt: int = 8192, batch: int = 128, context: int = 2048, steps: int = 20) -> dict:
    from tokenweave_b200 import LLM, SamplingParams, ops
    blocks = max(prompt // 128 + 2, batch * ((context + 2 * steps) // 128 + 2)) + 8
    llm = LLM(cfg, device="cuda", skip_tokenizer_init=True, load_format="dummy", max_num_batched_tokens=8192,
              max_num_seqs=batch, block_size=128, num_gpu_blocks_override=blocks, tokenweave_cuda_graphs=True, seed=0)
    runner = llm.llm_engine.core.executor.worker.runner
    g = torch.Generator().manual_seed(1)
    ids = lambda n: torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    one = SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True)

    def timed(prompts, sp):
        runner.timing_events = []
        flush.zero_()
        llm.generate(prompts, sp)
        torch.cuda.synchronize()
        ev, runner.timing_events = runner.timing_events, None
        return [a.elapsed_time(b) for a, b in ev]
    for _ in range(4):
        timed([ids(prompt)], one)
    pre = statistics.median(sum(timed([ids(prompt)], one)) for _ in range(5))
    many = SamplingParams(temperature=0.0, max_tokens=2 * steps, ignore_eos=True)
    dec = statistics.median(timed([ids(context) for _ in range(batch)], many)[-steps:])
    ops.check_status()
    llm.shutdown()
    torch.cuda.empty_cache()
    return {"prefill_tokens_per_s": prompt / pre * 1e3, "prefill_ms": pre, "decode_tokens_per_s": batch / dec * 1e3,
            "decode_ms_per_step": dec}


# ---- kernels -----------------------------------------------------------------------------------------------------------
class Timer:
    def __init__(self, iters: int = 9):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
        self.iters = iters
        self.rows: list[dict] = []
        self.bw, self.fl = peaks()

    def __call__(self, kernel: str, like: str, fn, nbytes: float, flops: float = 0.0) -> None:
        for _ in range(3):
            fn()
        ms = []
        for _ in range(self.iters):
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            b.synchronize()
            ms.append(a.elapsed_time(b))
        us = statistics.median(ms) * 1e3
        roof = max(nbytes / self.bw, flops / self.fl) * 1e6
        self.rows.append({"kernel": kernel, "like": like, "us": round(us, 2), "roofline_us": round(roof, 2),
                          "fraction": round(roof / us, 3)})
        torch.cuda.empty_cache()


def _r(*shape, scale=1.0):
    return (torch.randn(*shape, device="cuda") * scale).to(torch.bfloat16)


def _i(x):
    return torch.as_tensor(x, dtype=torch.int32, device="cuda")


def kernels(width: int, T: int = 8192, batch: int = 128, context: int = 2048) -> list[dict]:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    from tokenweave_b200.ops import reference
    heads, R, Q, ff, mh, groups = SIZES[width]
    t = Timer()
    row, inner = hops.latent_row(R, ROT), mh * P
    chan = inner + 2 * groups * N
    hkv = heads // 4
    cs = reference.build_cos_sin_cache(128, 16384, 500000.0, None, "cuda")
    cs_rot = reference.build_cos_sin_cache(ROT, 16384, 500000.0, None, "cuda")
    page, nb = 128, max(T // 128, batch * context // 128) + 8

    for m, tag in ((T, "prefill"), (batch, "decode")):
        w, w2 = _r(width), _r(width)
        x, res, x32, xa = _r(m, width), _r(m, width), torch.randn(m, width, device="cuda"), _r(m, width)
        t(f"postnorm_add [{tag}]", f"add_rmsnorm [{tag}]", lambda: hops.postnorm_add_(x, x32, w, 1e-5, xa), m * width * 12)
        t(f"add_rmsnorm [{tag}]", "", lambda: ops.add_rmsnorm_(x, res, w2, 1e-5), m * width * 8)
        z, o, coef = _r(m, ff), _r(m, ff), _r(4)
        t(f"polynorm [{tag}]", f"swiglu [{tag}]", lambda: hops.polynorm(z, coef, 1e-5, o, ff), m * ff * 4)
        gu = _r(m, 2 * ff)
        t(f"swiglu [{tag}]", "", lambda: ops.swiglu(gu, out=o), m * ff * 6)
        y, zz, wn, o2 = _r(m, inner), _r(m, inner), _r(inner), _r(m, inner)
        t(f"gated_group_norm [{tag}]", f"add_rmsnorm [{tag}]",
          lambda: hops.gated_group_norm(y, zz, wn, groups, 1e-5, o2), m * inner * 6)
        del gu, z, o
        # latent projections, rotation, cache write
        q8, kv8 = Q, (R + ROT + 7) // 8 * 8
        pr, cq, wq, wkv = _r(m, q8 + kv8 + heads * VDIM), _r(m, Q), _r(Q), _r(R)
        cache = torch.zeros(nb, page, row, dtype=torch.bfloat16, device="cuda")
        pos, slots = _i(range(m)), _i(range(128, 128 + m))
        t(f"latent_prep [{tag}]", f"rope_kv_write [{tag}]",
          lambda: hops.latent_prep(pr, 0, Q, wq, cq, q8, R, wkv, ROT, ROT, cs_rot, pos, slots, cache, 1e-5),
          m * (2 * Q + 2 * (R + ROT)) * 2)
        qkv = _r(m, (heads + 2 * hkv) * 128)
        kc, vc = (torch.zeros(m // page + 4, page, hkv, 128, dtype=torch.bfloat16, device="cuda") for _ in range(2))
        t(f"rope_kv_write [{tag}]", "", lambda: ops.rope_kv_write_(qkv, pos, slots, cs, kc, vc, heads, hkv, 128),
          m * (2 * heads + 4 * hkv) * 128 * 2)
        # state-space convolution
        xbc, xo = _r(m, chan), _r(m, chan)
        cw, cb, cst = _r(TAPS, chan), _r(chan), _r(batch, TAPS - 1, chan)
        single = tag == "decode"
        cu = _i(range(m + 1)) if single else _i([0, m])
        kvl = _i([context] * m) if single else _i([m])
        sl = _i(range(m)) if single else _i([0])
        rs = _i(range(m)) if single else _i([0] * m)
        t(f"causal_conv [{tag}]", f"rope_kv_write [{tag}]",
          lambda: hops.causal_conv(xbc, cw, cb, cst, xo, rs, cu, kvl, sl, single),
          m * chan * 4 + (m * 2 * (TAPS - 1) * chan * 2 if single else 0))
        # recurrence
        dt, bias, A, D = _r(m, mh), _r(mh, scale=0.1), _r(mh, scale=0.1), _r(mh)
        st = torch.randn(batch if single else 1, mh, P, N, device="cuda")
        ys = _r(m, inner)
        if single:
            seqs = _i(range(m))
            t("ssd_scan [decode]", "attn_decode", lambda: hops.ssd_scan(xbc, dt, bias, A, D, st, ys, seqs, cu, kvl, sl, groups),
              m * (mh * P * N * 8 + chan * 2 + inner * 2))
        else:
            seqs = _i([0])
            t("ssd_chunk [prefill]", "attn_prefill",
              lambda: hops.ssd_chunk(xbc, dt, bias, A, D, st, ys, seqs, cu, kvl, sl, groups),
              m * (chan + inner) * 2 + mh * P * N * 8, 2.0 * m * mh * (64 * N / (mh / groups) / 2 + 64 * P / 2 + 2 * N * P))
        del pr, qkv, xbc, xo, st, ys
        # matrix products, both models' shapes go through the same kernel
        for name, n, k, like in (("in_proj (latent)", q8 + kv8 + heads * VDIM, width, "qkv"),
                                 ("in_proj (mamba)", inner + chan + mh, width, "gate_up"),
                                 ("up_proj", ff, width, "gate_up"), ("down_proj", width, ff, "down")):
            a, b = _r(m, k), _r(n + (-n) % 8, k, scale=0.02)
            c = torch.empty(m, b.shape[0], dtype=torch.bfloat16, device="cuda")
            t(f"gemm {name} [{tag}]", f"gemm llama {like} [{tag}]", lambda: ops.gemm(a, b, out=c), (m * k + n * k + m * n) * 2,
              2.0 * m * n * k)
        lf = ff * 2 // 3 // 64 * 64
        for name, n, k in (("qkv", (heads + 2 * hkv) * 128, width), ("down", width, lf)):
            a, b = _r(m, k), _r(n, k, scale=0.02)
            c = torch.empty(m, n, dtype=torch.bfloat16, device="cuda")
            t(f"gemm llama {name} [{tag}]", "", lambda: ops.gemm(a, b, out=c), (m * k + n * k + m * n) * 2, 2.0 * m * n * k)
        a, b = _r(m, width), _r(2 * lf, width, scale=0.02)
        t(f"gemm llama gate_up [{tag}]", "", lambda: ops.gemm(a, b, swiglu=True), (m * width + 2 * lf * width + m * lf) * 2,
          4.0 * m * lf * width)
    _attention(t, heads, hkv, R, row, T, batch, context, page, nb, cs_rot)
    return t.rows


def _attention(t, heads, hkv, R, row, T, batch, context, page, nb, cs_rot) -> None:
    from tokenweave_b200 import ops
    from tokenweave_b200.ops import hybrid as hops
    scale = (DIM + ROT) ** -0.5
    # prefill of one sequence
    tiles = T // 128
    cu, kvl, ts = _i([0, T]), _i([T]), _i([0] * tiles)
    tq = _i(list(reversed(range(0, T, 128))))
    q, kv, lat = _r(T, heads * (DIM + ROT)), _r(T, heads * (DIM + VDIM)), _r(T, row)
    out, gate, begin = _r(T, heads * VDIM), _r(T, heads * VDIM), _i([0])
    t("latent_prefill", "attn_prefill",
      lambda: hops.latent_prefill(q, kv, lat, R, T, begin, out, gate, cu, kvl, ts, tq, tiles, heads, DIM, ROT, VDIM, scale),
      (q.numel() + kv.numel() + 2 * out.numel()) * 2, 2.0 * heads * T * T / 2 * (DIM + ROT + VDIM))
    pos = _i(range(T))
    t("rope_tail", "rope_kv_write [prefill]", lambda: hops.rope_tail_(q, heads, DIM + ROT, DIM, ROT, cs_rot, pos),
      T * heads * ROT * 4)
    bt = _i(range(1, T // page + 1)).view(1, -1)
    cache = _r(nb, page, row)
    cc = _i([0, T])
    t("latent_gather", "gather_cache", lambda: hops.latent_gather(cache, begin, cc, T, bt, lat), T * row * 4)
    kc, vc = _r(nb, page, hkv, 128), _r(nb, page, hkv, 128)
    lo = torch.empty(T, hkv, 128, dtype=torch.bfloat16, device="cuda")
    t("gather_cache", "", lambda: ops.gather_cache(kc, bt, cc, T, out=lo), T * hkv * 128 * 4)
    wkv, kvo = _r(heads * (DIM + VDIM), R, scale=0.04), torch.empty_like(kv)
    t("gemm ukv_proj (expand)", "gemm llama gate_up [prefill]", lambda: ops.gemm(lat[:, :R], wkv, out=kvo),
      (T * R + wkv.numel() + kvo.numel()) * 2, 2.0 * T * R * heads * (DIM + VDIM))
    qq, oo = _r(T, heads * 128), _r(T, heads * 128)
    t("attn_prefill", "", lambda: ops.attn_prefill(qq, kc, vc, oo, cu, kvl, bt, ts, tq, tiles, heads, hkv, 128, 128 ** -0.5),
      (2 * qq.numel() + 2 * T * hkv * 128) * 2, 2.0 * heads * T * T / 2 * 256)
    del q, kv, out, gate, qq, oo, kvo
    # decode of a batch
    n, per = batch, context // page
    btd = _i([[1 + b * per + j for j in range(per)] for b in range(n)])
    tok, lens = _i(range(n)), _i([context] * n)
    qa, o = _r(n, heads, row), _r(n, heads, R)
    t("latent_decode", "attn_decode",
      lambda: hops.latent_attention(qa, cache, tok, lens, n, btd, R, scale, o, context),
      n * context * row * 2 + qa.numel() * 2 + o.numel() * 2, 2.0 * n * heads * context * (row + R))
    qd, od = _r(n, heads * 128), _r(n, heads * 128)
    t("attn_decode", "", lambda: ops.attn_decode(qd, kc, vc, od, tok, tok, lens, n, btd, heads, hkv, 128, 128 ** -0.5, context),
      n * context * hkv * 128 * 4 + 4 * qd.numel(), 2.0 * n * heads * context * 256)
    q, ukt = _r(n, heads * (DIM + ROT)), _r(heads, R, DIM, scale=0.09)
    t("latent_absorb (head_gemm + latent_query)", "gemm llama gate_up [decode]",
      lambda: hops.latent_absorb(q, tok, ukt, heads, DIM, ROT, ROT, R, cs_rot, lens, qa),
      (q.numel() + ukt.numel() + qa.numel()) * 2, 2.0 * n * heads * DIM * R)
    uv, g, at = _r(heads, VDIM, R, scale=0.04), _r(n, heads * VDIM), _r(n, heads * VDIM)
    t("latent_values (head_gemm + gate)", "gemm llama gate_up [decode]",
      lambda: hops.latent_values(o, tok, uv, heads, VDIM, R, g, at), (o.numel() + uv.numel() + 2 * at.numel()) * 2,
      2.0 * n * heads * VDIM * R)


def with_ratios(rows: list[dict]) -> list[dict]:
    """Adds to every row how much further it is from its roofline than the like kernel."""
    frac = {r["kernel"]: r["fraction"] for r in rows}
    for r in rows:
        if r["like"]:
            r["like_fraction"] = frac[r["like"]]
            r["distance_ratio"] = round(frac[r["like"]] / r["fraction"], 2)
    return rows


def run(sizes=None, steps: int = 20) -> dict:
    out = {}
    for width in sizes or SIZES:
        hybrid, llama = models(width)
        rows = with_ratios(kernels(width))
        out[str(width)] = {"hybrid": throughput(hybrid, steps=steps), "llama": throughput(llama, steps=steps), "kernels": rows}
    return out


def print_tables(result: dict, names: tuple) -> None:
    for width, res in result.items():
        print(f"== width {width}")
        for name in names:
            print(f"{name:8s}" + "  ".join(f"{k} {v:.1f}" for k, v in res[name].items()))
        for r in res["kernels"]:
            print(f"{r['kernel']:52s} {r['us']:9.1f} us  roofline {r['roofline_us']:8.1f}  {r['fraction']:.2f}"
                  + (f"   like {r['like']} {r['like_fraction']:.2f}  x{r['distance_ratio']:.2f}" if r["like"] else ""))


if __name__ == "__main__":
    print_tables(run(), ("hybrid", "llama"))

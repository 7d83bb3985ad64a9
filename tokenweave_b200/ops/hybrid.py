"""Operators of models whose layers mix attention and recurrences and whose residual stream is fp32: latent attention
over a paged latent cache, the state-space (Mamba-2) recurrence with its convolution, the norm of a sublayer's output
added to the residual, and the polynomial-norm activation; for blocks whose sublayers read one norm of the stream,
grouped attention with its options (query and key norms, short convolution, rotation, query temperature, distance bias,
sink, sliding window, sigmoid weights in chunks), lightning attention, embeddings with token pairs, and the fused projections;
hyper-connections; norms on both sides of a sublayer with averages over the depth; the minGRU recurrence.

Like the other operators, CUDA tensors (bf16 or fp32) go to the kernels of ``_C.so`` and CPU tensors to plain PyTorch
(:mod:`.reference_hybrid`). ``meta`` below is the step's :class:`~tokenweave_b200.layers.attention.AttentionMetadata`.
"""
from __future__ import annotations

from typing import Optional

import torch

from . import _native, reference_hybrid as ref
from . import COL_ACTS, _p, _row_stride, _stream, decode_splits_tc, gemm, status_word


def _dt(*ts: Optional[torch.Tensor]) -> int:
    """The launchers' dtype code; every tensor must be stored in the same type."""
    kinds = {t.dtype for t in ts if t is not None}
    if len(kinds) != 1 or next(iter(kinds)) not in (torch.bfloat16, torch.float32):
        raise TypeError(f"expected tensors of one type, bfloat16 or float32, got {sorted(map(str, kinds))}")
    return 0 if next(iter(kinds)) == torch.bfloat16 else 1


# ---- residual stream and row-wise kernels ------------------------------------------------------------------
def embed_residual(ids: torch.Tensor, table: torch.Tensor, x32: torch.Tensor, xa: torch.Tensor, width: int) -> None:
    """``x32 = table[ids]`` (fp32 residual stream) and ``xa`` the same rows in the activation type."""
    if not table.is_cuda:
        ref.embed_residual(ids, table, x32, xa, width)
        return
    assert ids.dtype == torch.int32 and x32.dtype == torch.float32
    _native.call("tw_embed_residual", ids.data_ptr(), table.data_ptr(), _row_stride(table), x32.data_ptr(),
                 _row_stride(x32), xa.data_ptr(), _row_stride(xa), ids.shape[0], width, table.shape[0], _dt(table, xa),
                 _stream())


def postnorm_add_(y: torch.Tensor, x32: torch.Tensor, weight: torch.Tensor, eps: float, xa: torch.Tensor,
                  final_weight: Optional[torch.Tensor] = None) -> None:
    """``x32 += rmsnorm(y) * weight`` and ``xa = x32`` (in the activation type); behind the last layer, with
    ``final_weight``, ``xa = rmsnorm(x32) * final_weight``. The row width is the weight's length."""
    if not y.is_cuda:
        ref.postnorm_add_(y, x32, weight, eps, xa, final_weight)
        return
    assert x32.dtype == torch.float32
    _native.call("tw_postnorm_add", y.data_ptr(), _row_stride(y), x32.data_ptr(), _row_stride(x32), weight.data_ptr(),
                 xa.data_ptr(), _row_stride(xa), _p(final_weight), y.shape[0], weight.numel(), float(eps),
                 _dt(y, weight, xa, final_weight), _stream())


def polynorm(z: torch.Tensor, coef: torch.Tensor, eps: float, out: torch.Tensor, width: int) -> torch.Tensor:
    """``a N(z) + b N(z^2) + c N(z^3) + e`` with ``coef = (a, b, c, e)`` and N dividing a row by its root mean square."""
    if not z.is_cuda:
        out[:, :width] = ref.polynorm(z[:, :width], coef, eps)
        return out
    _native.call("tw_polynorm", z.data_ptr(), _row_stride(z), coef.data_ptr(), out.data_ptr(), _row_stride(out),
                 z.shape[0], width, float(eps), _dt(z, coef, out), _stream())
    return out


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, groups: int, eps: float,
                     out: torch.Tensor) -> torch.Tensor:
    """RMS norm of ``y * silu(z)`` in ``groups`` equal parts of the row, times ``weight`` (the gate comes first)."""
    c = weight.numel()
    if not y.is_cuda:
        out[:, :c] = ref.gated_group_norm(y[:, :c], z[:, :c], weight, groups, eps)
        return out
    _native.call("tw_gated_group_norm", y.data_ptr(), _row_stride(y), z.data_ptr(), _row_stride(z), weight.data_ptr(),
                 out.data_ptr(), _row_stride(out), y.shape[0], c, groups, float(eps), _dt(y, z, weight, out), _stream())
    return out


# ---- hyper-connections: several residual streams ---------------------------------------------------------------
# ``x``: fp32 [T, streams, padded width]; ``hc``: a sublayer's coefficients {"in" [S], "out" [S], "mix" [S, S] (from, to)}
# in fp32; norm weights are stored around ``offset``.
def embed_streams(ids: torch.Tensor, table: torch.Tensor, x: torch.Tensor, hc_in: torch.Tensor, weight: torch.Tensor,
                  offset: float, eps: float, xa: torch.Tensor) -> None:
    """The first stream ``= table[ids]`` (all begin as that row: the first :func:`streams_step` is told so);
    ``xa = rmsnorm(sum_s in[s] x_0) * (offset + weight)``."""
    if not table.is_cuda:
        ref.embed_streams(ids, table, x, hc_in, weight, offset, eps, xa)
        return
    assert ids.dtype == torch.int32 and x.dtype == hc_in.dtype == torch.float32 and x.stride(2) == 1
    _native.call("tw_embed_streams", ids.data_ptr(), table.data_ptr(), _row_stride(table), table.shape[0], x.data_ptr(),
                 x.stride(0), x.stride(1), x.shape[1], hc_in.data_ptr(), weight.data_ptr(), float(offset), xa.data_ptr(),
                 _row_stride(xa), ids.shape[0], weight.numel(), float(eps), _dt(table, weight, xa), _stream())


def streams_step(y: torch.Tensor, x: torch.Tensor, hc: dict, mult: float, next_in: Optional[torch.Tensor],
                 weight: torch.Tensor, offset: float, eps: float, xa: torch.Tensor, first: bool = False) -> None:
    """``x_t <- sum_s mix[s, t] x_s + mult out[t] y`` (from the old streams), then the next sublayer's input
    ``xa = rmsnorm(sum_s next_in[s] x_s) * (offset + weight)``. ``next_in`` None: behind the last sublayer - the norm of the
    streams' sum, the streams themselves are not stored. ``first``: every old stream is the first one."""
    if not y.is_cuda:
        ref.streams_step(y, x, hc, mult, next_in, weight, offset, eps, xa, first)
        return
    assert x.dtype == hc["mix"].dtype == hc["out"].dtype == torch.float32 and x.stride(2) == 1
    assert next_in is None or next_in.dtype == torch.float32
    _native.call("tw_streams_step", y.data_ptr(), _row_stride(y), x.data_ptr(), x.stride(0), x.stride(1), x.shape[1],
                 hc["mix"].data_ptr(), hc["out"].data_ptr(), float(mult), _p(next_in), int(first), int(next_in is not None),
                 weight.data_ptr(), float(offset), xa.data_ptr(), _row_stride(xa), y.shape[0], weight.numel(), float(eps),
                 _dt(y, weight, xa), _stream())


# ---- norms on both sides of a sublayer, averages over the depth -------------------------------------------------
# A norm is a pair (weight, bias): a layer norm, or (weight, None): an RMS norm. ``results``: fp32 [layers, T, padded width],
# the embedding output and the layers' results in order.
def embed_sandwich(ids: torch.Tensor, table: torch.Tensor, scale: float, x32: torch.Tensor, first: Optional[torch.Tensor],
                   norm: tuple, eps: float, xa: torch.Tensor) -> None:
    """``x32 = scale * table[ids]``; ``first``: a copy of it; ``xa`` its norm."""
    w, b = norm
    if not table.is_cuda:
        ref.embed_sandwich(ids, table, scale, x32, first, norm, eps, xa)
        return
    assert ids.dtype == torch.int32 and x32.dtype == torch.float32 and (first is None or first.dtype == torch.float32)
    _native.call("tw_embed_sandwich", ids.data_ptr(), table.data_ptr(), _row_stride(table), table.shape[0], float(scale),
                 x32.data_ptr(), _row_stride(x32), _p(first), _row_stride(first) if first is not None else 0, w.data_ptr(),
                 _p(b), int(b is not None), xa.data_ptr(), _row_stride(xa), ids.shape[0], w.numel(), float(eps),
                 _dt(table, w, b, xa), _stream())


def sandwich_step(y: torch.Tensor, x32: torch.Tensor, post: tuple, nxt: tuple, eps: float, xa: torch.Tensor,
                  coef: Optional[torch.Tensor] = None, results: Optional[torch.Tensor] = None, last: bool = False) -> None:
    """``x32 += norm_post(y)``; behind a layer, with ``coef`` (fp32 [n + 1]): the sum is result n (kept in ``results[n]``,
    unless ``last``) and ``x32 = sum_j coef[j] results[j]``; then ``xa = norm_next(x32)``. ``last``: behind the last sublayer,
    the stream itself is not stored."""
    (w, b), (wn, bn) = post, nxt
    if (b is None) != (bn is None):
        raise ValueError("norms of one kind are needed")
    n = coef.numel() - 1 if coef is not None else 0
    if not y.is_cuda:
        ref.sandwich_step(y, x32, post, nxt, eps, xa, coef, results, last)
        return
    assert x32.dtype == torch.float32 and (coef is None or (coef.dtype == results.dtype == torch.float32
                                                            and results.stride(2) == 1 and results.shape[0] >= n + (not last)))
    keep = results[n] if coef is not None and not last else None
    ldp, lds = (results.stride(1), results.stride(0)) if coef is not None else (0, 0)
    _native.call("tw_sandwich_step", y.data_ptr(), _row_stride(y), x32.data_ptr(), _row_stride(x32), int(not last),
                 w.data_ptr(), _p(b), _p(results) if coef is not None else None, ldp, lds, n, _p(coef), _p(keep),
                 wn.data_ptr(), _p(bn), int(b is not None), xa.data_ptr(), _row_stride(xa), y.shape[0], w.numel(), float(eps),
                 _dt(y, w, b, wn, bn, xa), _stream())


# ---- minGRU -----------------------------------------------------------------------------------------------------
def min_gru(p: torch.Tensor, bz: torch.Tensor, bx: torch.Tensor, state: torch.Tensor, out: torch.Tensor, seqs: torch.Tensor,
            cu_q: torch.Tensor, kv_lens: torch.Tensor, slots: torch.Tensor, chunked: bool = False) -> None:
    """Per channel ``z = sigmoid(pz + bz)``, ``u = px + bx``, ``S <- (1 - z) S + z (u + 1/2 if u >= 0 else sigmoid(u))``,
    ``out = S silu(pg)`` of the listed sequences; ``p`` rows are [pz | px | pg], each as wide as ``state`` (fp32 [slots,
    channels, a multiple of eight]). ``chunked``: many tokens at a time (long runs)."""
    if seqs.shape[0] == 0:
        return
    if not p.is_cuda:
        ref.min_gru(p, bz, bx, state, out, seqs, cu_q, kv_lens, slots)
        return
    assert state.dtype == bz.dtype == bx.dtype == torch.float32
    _native.call("tw_min_gru", p.data_ptr(), _row_stride(p), bz.data_ptr(), bx.data_ptr(), state.data_ptr(), out.data_ptr(),
                 _row_stride(out), seqs.data_ptr(), seqs.shape[0], cu_q.data_ptr(), kv_lens.data_ptr(), slots.data_ptr(),
                 state.shape[1], int(chunked), _dt(p, out), _stream())


# ---- latent attention -----------------------------------------------------------------------------------------
def latent_row(kv_rank: int, rot: int) -> int:
    """Elements of a latent cache row: the latent and the rotated key part, each padded to eight."""
    return (kv_rank + 7) // 8 * 8 + (rot + 7) // 8 * 8


def latent_prep(p: torch.Tensor, q_off: int, q_rank: int, wq: torch.Tensor, cq: torch.Tensor, kv_off: int, kv_rank: int,
                wkv: torch.Tensor, rot: int, rot_dims: int, cos_sin: torch.Tensor, positions: torch.Tensor,
                slots: torch.Tensor, cache: torch.Tensor, eps: float) -> None:
    """Norms of the two latents in the packed projection rows ``p``, rotation of the shared key part, cache write.
    ``cache``: [blocks, page, row]."""
    if not p.is_cuda:
        ref.latent_prep(p, q_off, q_rank, wq, cq, kv_off, kv_rank, wkv, rot, rot_dims, cos_sin, positions, slots, cache,
                        eps)
        return
    _native.call("tw_latent_prep", p.data_ptr(), _row_stride(p), q_off, q_rank, wq.data_ptr(), cq.data_ptr(),
                 _row_stride(cq), kv_off, kv_rank, wkv.data_ptr(), rot, rot_dims, cos_sin.data_ptr(),
                 positions.data_ptr(), slots.data_ptr(), cache.data_ptr(), cache.shape[-1], p.shape[0], float(eps),
                 _dt(p, wq, cq, wkv, cache), _stream())


def rope_tail_(q: torch.Tensor, heads: int, head_stride: int, off: int, rot_dims: int, cos_sin: torch.Tensor,
               positions: torch.Tensor) -> None:
    """Rotates elements ``[off, off + rot_dims)`` of every head of every row in place (CUDA; the un-absorbed form)."""
    _native.call("tw_rope_tail", q.data_ptr(), _row_stride(q), q.shape[0], heads, head_stride, off, rot_dims,
                 cos_sin.data_ptr(), positions.data_ptr(), _dt(q), _stream())


def latent_absorb(q: torch.Tensor, rows: torch.Tensor, w_ukt: torch.Tensor, heads: int, dim: int, rot: int,
                  rot_dims: int, kv_rank: int, cos_sin: torch.Tensor, positions: torch.Tensor, qa: torch.Tensor) -> None:
    """Absorbed queries ``qa`` [n, heads, row] of the listed rows of ``q`` ([T, heads * (dim + rot)]): the key map
    ``w_ukt`` [heads, kv_rank, >= dim] applied to the unrotated part, the rotated part, zero pads."""
    n = rows.shape[0]
    if not q.is_cuda:
        qa[:n] = ref.latent_absorb(q, rows, w_ukt, heads, dim, rot, rot_dims, kv_rank, cos_sin, positions, qa.shape[-1])
        return
    dt = _dt(q, w_ukt, qa)
    row = qa.shape[-1]
    _native.call("tw_head_gemm", q.data_ptr(), _row_stride(q), dim + rot, rows.data_ptr(), w_ukt.data_ptr(),
                 w_ukt.stride(0), w_ukt.stride(1), qa.data_ptr(), heads * row, row, None, None, 0, 0, heads, n, kv_rank,
                 dim, dt, _stream())
    _native.call("tw_latent_query", q.data_ptr(), _row_stride(q), rows.data_ptr(), n, qa.data_ptr(), heads, dim + rot,
                 dim, rot, rot_dims, kv_rank, row, cos_sin.data_ptr(), positions.data_ptr(), dt, _stream())


def _key_tiles(max_kv_len: int, window: int = 0, keep: int = 0) -> int:
    """Most 128-key tiles that hold visible keys of one row (``window``: of a window or a chunk)."""
    tiles = (max_kv_len + 127) // 128
    return min(tiles, (window + 126) // 128 + 1 + (keep + 127) // 128) if window else tiles


def latent_decode_plan(n: int, heads: int, row: int, kv_rank: int, page: int, dtype: torch.dtype, max_kv_len: int,
                       sm_count: int = 148, window: int = 0) -> tuple[str, int]:
    """(kernel, key splits) of an absorbed attention launch: "tc" (tensor cores: bf16, cache rows of up to 640 elements
    with a latent of up to 512) or "simt" (fp32 and every other size)."""
    if dtype != torch.bfloat16 or row > 640 or kv_rank > 512 or page < 8 or page > 128 or 128 % page:
        return "simt", 1
    blocks = (heads + 15) // 16 if heads <= 16 else (heads + 31) // 32
    return "tc", decode_splits_tc(n * blocks, _key_tiles(max_kv_len, window), sm_count)


_partials: dict[tuple, tuple[torch.Tensor, torch.Tensor]] = {}


def _partial_buffers(device, count: int, width: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Workspace of split launches; sizes are powers of two and buffers are never freed (captured graphs keep their
    addresses)."""
    count = 1 << max(0, (count - 1).bit_length())
    key = (device.index, count, width)
    ws = _partials.get(key)
    if ws is None:
        ws = _partials[key] = (torch.empty(count * width, dtype=torch.float32, device=device),
                               torch.empty(count * 2, dtype=torch.float32, device=device))
    return ws


def latent_attention(qa: torch.Tensor, cache: torch.Tensor, tok_seq: torch.Tensor, tok_kvlen: torch.Tensor, n: int,
                     block_table: torch.Tensor, kv_rank: int, scale: float, out: torch.Tensor, max_kv_len: int,
                     sm_count: int = 148, kernel: Optional[str] = None, window: int = 0,
                     sink: Optional[torch.Tensor] = None) -> None:
    """Causal attention of ``n`` absorbed query rows over the paged latent cache; ``out`` [n, heads, kv_rank].
    ``window`` > 0: a row sees the last ``window`` keys, itself among them (and the tensor-core kernels keep 16 bits of the
    softmax weights, 8 without it); ``sink`` (fp32 [heads]): exp(sink) joins the
    denominator. ``kernel``: force one of :func:`latent_decode_plan`'s kernels (tests)."""
    if n == 0:
        return
    heads, row, page = qa.shape[1], qa.shape[2], cache.shape[1]
    if not qa.is_cuda:
        out[:n] = ref.latent_attention(qa[:n], cache, tok_seq, tok_kvlen, block_table, kv_rank, scale, window, sink)
        return
    dt = _dt(qa, cache, out)
    assert sink is None or sink.dtype == torch.float32
    plan, splits = latent_decode_plan(n, heads, row, kv_rank, page, qa.dtype, max_kv_len, sm_count, window)
    if (kernel or plan) == "tc":
        po = pm = None
        if splits > 1:
            po, pm = _partial_buffers(qa.device, n * heads * splits, kv_rank)
        _native.call("tw_latent_decode", qa.data_ptr(), cache.data_ptr(), cache.shape[0], page, tok_seq.data_ptr(),
                     tok_kvlen.data_ptr(), n, block_table.data_ptr(), block_table.shape[1], out.data_ptr(), heads, row,
                     kv_rank, float(scale), int(window), _p(sink), int(window > 0), splits, _p(po), _p(pm),
                     status_word(qa.device).data_ptr(), _stream())
        return
    _native.call("tw_latent_attn", qa.data_ptr(), cache.data_ptr(), tok_seq.data_ptr(), tok_kvlen.data_ptr(), n,
                 block_table.data_ptr(), block_table.shape[1], page, out.data_ptr(), heads, row, kv_rank, float(scale),
                 int(window), _p(sink), dt, _stream())


def latent_expandable(dtype: torch.dtype, dim: int, rot: int, vdim: int) -> bool:
    """Head sizes the expanded tensor-core prefill takes (bf16)."""
    kc, vc = (dim + 63) // 64 + (rot + 63) // 64, (vdim + 63) // 64
    return dtype == torch.bfloat16 and dim % 8 == rot % 8 == vdim % 8 == 0 and vc <= 2 and kc + vc <= 5


def latent_prefill(q: torch.Tensor, kv: torch.Tensor, latents: torch.Tensor, rot_off: int, ctx_rows: int,
                   ctx_begin: torch.Tensor, out: torch.Tensor, gate: Optional[torch.Tensor], cu_q: torch.Tensor,
                   kv_lens: torch.Tensor, tile_seq: torch.Tensor, tile_q0: torch.Tensor, num_tiles: int, heads: int,
                   dim: int, rot: int, vdim: int, scale: float, window: int = 0,
                   sink: Optional[torch.Tensor] = None) -> None:
    """Expanded causal attention of the listed 128-query tiles (CUDA, bf16). ``q`` [T, heads * (dim + rot)] with rotated
    tails; ``kv`` [ctx_rows, heads * dim | heads * vdim] and the rotated part ``latents[:, rot_off:]`` of every
    context row; key k of sequence b is workspace row ``ctx_begin[b] + k``. ``window`` and ``sink`` as for
    :func:`latent_attention`."""
    _dt(q, kv, latents, out, gate)
    kr = latents[:, rot_off:]
    _native.call("tw_latent_prefill", q.data_ptr(), _row_stride(q), q.shape[0], kv.data_ptr(), _row_stride(kv),
                 kr.data_ptr(), _row_stride(kr), ctx_rows, ctx_begin.data_ptr(), out.data_ptr(), _row_stride(out),
                 _p(gate), _row_stride(gate) if gate is not None else 0, cu_q.data_ptr(), kv_lens.data_ptr(),
                 tile_seq.data_ptr(), tile_q0.data_ptr(), num_tiles, heads, dim, rot, vdim, float(scale), int(window),
                 _p(sink), status_word(q.device).data_ptr(), _stream())


def latent_values(o: torch.Tensor, rows: torch.Tensor, w_uv: torch.Tensor, heads: int, vdim: int, kv_rank: int,
                  gate: Optional[torch.Tensor], out: torch.Tensor) -> None:
    """``out[rows, h * vdim : ] = (w_uv[h] o[:, h]) * sigmoid(gate)``: head values of the weighted latents. ``w_uv``:
    [heads, vdim, >= kv_rank]; ``gate`` (or None) and ``out`` are rows of all tokens of the step."""
    n = rows.shape[0]
    if not o.is_cuda:
        ref.latent_values(o[:n], rows, w_uv, heads, vdim, kv_rank, gate, out)
        return
    _native.call("tw_head_gemm", o.data_ptr(), heads * kv_rank, kv_rank, None, w_uv.data_ptr(), w_uv.stride(0),
                 w_uv.stride(1), out.data_ptr(), _row_stride(out), vdim, rows.data_ptr(), _p(gate),
                 _row_stride(gate) if gate is not None else 0, vdim, heads, n, vdim, kv_rank, _dt(o, w_uv, out, gate),
                 _stream())


def latent_gather(cache: torch.Tensor, seqs: torch.Tensor, cu: torch.Tensor, max_rows: int, block_table: torch.Tensor,
                  out: torch.Tensor, first: Optional[torch.Tensor] = None) -> None:
    """``cu[i + 1] - cu[i]`` cache rows of sequence ``seqs[i]``, in order from key ``first[i]`` (None: 0) on, into
    ``out[cu[i]:]`` (CUDA)."""
    _native.call("tw_latent_gather", cache.data_ptr(), out.data_ptr(), seqs.data_ptr(), cu.data_ptr(), _p(first),
                 seqs.shape[0], max_rows, block_table.data_ptr(), block_table.shape[1], cache.shape[1],
                 cache.shape[2] * cache.element_size(), _stream())


# ---- state-space recurrence -------------------------------------------------------------------------------------
def causal_conv(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, state: torch.Tensor, out: torch.Tensor,
                row_seq: torch.Tensor, cu_q: torch.Tensor, kv_lens: torch.Tensor, slots: torch.Tensor,
                single: bool) -> None:
    """Per-channel causal convolution + bias + silu of the step's rows; ``weight`` [taps, channels] (last tap = current
    token), ``state`` [slots, taps - 1, channels] is read for the inputs before a sequence's rows and moved on.
    ``single``: every sequence has exactly one row."""
    taps, channels = weight.shape
    if not x.is_cuda:
        ref.causal_conv(x, weight, bias, state, out, cu_q, kv_lens, slots)
        return
    _native.call("tw_causal_conv", x.data_ptr(), _row_stride(x), weight.data_ptr(), bias.data_ptr(), state.data_ptr(),
                 out.data_ptr(), _row_stride(out), row_seq.data_ptr(), cu_q.data_ptr(), kv_lens.data_ptr(),
                 slots.data_ptr(), x.shape[0], cu_q.shape[0] - 1, channels, taps, int(single),
                 _dt(x, weight, bias, state, out), _stream())


def ssd_scan(xbc: torch.Tensor, dt: torch.Tensor, dt_bias: torch.Tensor, A_log: torch.Tensor, D: torch.Tensor,
             state: torch.Tensor, y: torch.Tensor, seqs: torch.Tensor, cu_q: torch.Tensor, kv_lens: torch.Tensor,
             slots: torch.Tensor, groups: int) -> None:
    """Token-by-token state-space recurrence of the listed sequences. ``state``: fp32 [slots, heads, vdim, state]."""
    if seqs.shape[0] == 0:
        return
    _, heads, vdim, N = state.shape
    if not xbc.is_cuda:
        ref.ssd_scan(xbc, dt, dt_bias, A_log, D, state, y, seqs, cu_q, kv_lens, slots, groups)
        return
    assert state.dtype == torch.float32
    _native.call("tw_ssd_scan", xbc.data_ptr(), _row_stride(xbc), dt.data_ptr(), _row_stride(dt), dt_bias.data_ptr(),
                 A_log.data_ptr(), D.data_ptr(), state.data_ptr(), y.data_ptr(), _row_stride(y), seqs.data_ptr(),
                 seqs.shape[0], cu_q.data_ptr(), kv_lens.data_ptr(), slots.data_ptr(), heads, vdim, N, groups,
                 _dt(xbc, dt, dt_bias, A_log, D, y), _stream())


CHUNK_MIN_TOKENS = 16        # runs of at least this many tokens take the chunked form


def ssd_chunkable(dtype: torch.dtype, vdim: int, N: int) -> bool:
    """Sizes the chunked tensor-core form of the recurrence takes (bf16 activations)."""
    return dtype == torch.bfloat16 and vdim % 8 == 0 and N % 8 == 0 and N <= 256


def ssd_chunk(xbc: torch.Tensor, dt: torch.Tensor, dt_bias: torch.Tensor, A_log: torch.Tensor, D: torch.Tensor,
              state: torch.Tensor, y: torch.Tensor, seqs: torch.Tensor, cu_q: torch.Tensor, kv_lens: torch.Tensor,
              slots: torch.Tensor, groups: int, form: int = 0) -> None:
    """:func:`ssd_scan` for long runs, many tokens at a time on the tensor cores (CUDA, bf16). ``form`` 0: tcgen05 in
    chunks of 128 for states of up to 128 dimensions, warp-level products in chunks of 64 beyond; 1: always the latter."""
    if seqs.shape[0] == 0:
        return
    _, heads, vdim, N = state.shape
    assert state.dtype == torch.float32 and _dt(xbc, dt, dt_bias, A_log, D, y) == 0
    _native.call("tw_ssd_chunk", xbc.data_ptr(), _row_stride(xbc), xbc.shape[0], dt.data_ptr(), _row_stride(dt), dt_bias.data_ptr(),
                 A_log.data_ptr(), D.data_ptr(), state.data_ptr(), y.data_ptr(), _row_stride(y), seqs.data_ptr(),
                 seqs.shape[0], cu_q.data_ptr(), kv_lens.data_ptr(), slots.data_ptr(), heads, vdim, N, groups, form,
                 status_word(xbc.device).data_ptr(), _stream())


# ---- lightning attention: the recurrence with unit steps and a fixed decay per head --------------------------------
def decay_scan(p: torch.Tensor, decay: torch.Tensor, state: torch.Tensor, y: torch.Tensor, seqs: torch.Tensor,
               cu_q: torch.Tensor, kv_lens: torch.Tensor, slots: torch.Tensor) -> None:
    """``S <- decay[h] S + v k^T``, ``y = S q`` token by token; ``p`` rows are [v of all heads | k | q | ...]."""
    if seqs.shape[0] == 0:
        return
    _, heads, vdim, N = state.shape
    if not p.is_cuda:
        ref.decay_scan(p, decay, state, y, seqs, cu_q, kv_lens, slots)
        return
    assert state.dtype == decay.dtype == torch.float32
    _native.call("tw_decay_scan", p.data_ptr(), _row_stride(p), decay.data_ptr(), state.data_ptr(), y.data_ptr(),
                 _row_stride(y), seqs.data_ptr(), seqs.shape[0], cu_q.data_ptr(), kv_lens.data_ptr(), slots.data_ptr(),
                 heads, vdim, N, _dt(p, y), _stream())


def decay_chunk(p: torch.Tensor, decay: torch.Tensor, state: torch.Tensor, y: torch.Tensor, seqs: torch.Tensor,
                cu_q: torch.Tensor, kv_lens: torch.Tensor, slots: torch.Tensor, form: int = 0) -> None:
    """:func:`decay_scan` for long runs on the tensor cores (CUDA, bf16); ``form`` as for :func:`ssd_chunk`."""
    if seqs.shape[0] == 0:
        return
    _, heads, vdim, N = state.shape
    assert state.dtype == decay.dtype == torch.float32 and _dt(p, y) == 0
    _native.call("tw_decay_chunk", p.data_ptr(), _row_stride(p), p.shape[0], decay.data_ptr(), state.data_ptr(),
                 y.data_ptr(), _row_stride(y), seqs.data_ptr(), seqs.shape[0], cu_q.data_ptr(), kv_lens.data_ptr(),
                 slots.data_ptr(), heads, vdim, N, form, status_word(p.device).data_ptr(), _stream())


def norm_gate(y: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, count: int, eps: float, scale: float,
              out: torch.Tensor) -> None:
    """``out = rmsnorm(y) * weight * sigmoid(gate) * scale``; rows as wide as the weight, of which ``count`` elements are
    not padding (zeros)."""
    if not y.is_cuda:
        ref.norm_gate(y, gate, weight, count, eps, scale, out)
        return
    _native.call("tw_norm_gate", y.data_ptr(), _row_stride(y), gate.data_ptr(), _row_stride(gate), weight.data_ptr(),
                 out.data_ptr(), _row_stride(out), y.shape[0], weight.numel(), count, float(eps), float(scale),
                 _dt(y, gate, weight, out), _stream())


# ---- parallel blocks: embedding, sums and norms, projections ---------------------------------------------------------
def embed_norm(ids: torch.Tensor, table: torch.Tensor, pairs: Optional[torch.Tensor], spec: Optional[dict], meta,
               x32: torch.Tensor, first: Optional[torch.Tensor], weight: torch.Tensor, eps: float, xa: torch.Tensor) -> None:
    """``x32 = table[ids]``, plus the token pair's row of ``pairs`` (``spec`` = {"buckets", "mul_prev", "mul_cur"}: row
    ``(previous * mul_prev + token * mul_cur) mod buckets``, the last row for a sequence's first token); ``first``: a copy
    of that; ``xa = rmsnorm(x32) * weight``."""
    if not table.is_cuda:
        ref.embed_norm(ids, table, pairs, spec, meta, x32, first, weight, eps, xa)
        return
    assert ids.dtype == torch.int32 and x32.dtype == torch.float32
    row_seq = prev = None
    mul = (1, 0, 0)
    if pairs is not None:
        row_seq, prev = meta.extra["row_seq"], meta.extra["prev_token"]
        mul = tuple(int(spec[k]) for k in ("buckets", "mul_prev", "mul_cur"))
        assert pairs.shape[0] == mul[0] + 1
    _native.call("tw_embed_norm", ids.data_ptr(), table.data_ptr(), _row_stride(table), table.shape[0], _p(pairs),
                 _row_stride(pairs) if pairs is not None else 0, *mul, _p(row_seq), meta.cu_q.data_ptr(), _p(prev),
                 x32.data_ptr(), _row_stride(x32), _p(first), _row_stride(first) if first is not None else 0,
                 weight.data_ptr(), xa.data_ptr(), _row_stride(xa), ids.shape[0], weight.numel(), float(eps),
                 _dt(table, pairs, weight, xa), _stream())


def add_prenorm_(y: torch.Tensor, x32: torch.Tensor, first: Optional[torch.Tensor], weight: torch.Tensor, eps: float,
                 xa: torch.Tensor) -> None:
    """``x32 += y (+ first)``, ``xa = rmsnorm(x32) * weight``."""
    if not y.is_cuda:
        ref.add_prenorm_(y, x32, first, weight, eps, xa)
        return
    assert x32.dtype == torch.float32 and (first is None or first.dtype == torch.float32)
    _native.call("tw_add_prenorm", y.data_ptr(), _row_stride(y), x32.data_ptr(), _row_stride(x32), _p(first),
                 _row_stride(first) if first is not None else 0, weight.data_ptr(), xa.data_ptr(), _row_stride(xa),
                 y.shape[0], weight.numel(), float(eps), _dt(y, weight, xa), _stream())


def projection(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], cols: Optional[tuple[int, int]],
               out: torch.Tensor, act: str = "silu") -> torch.Tensor:
    """``out = x w^T + bias``, then ``act`` ("silu" or "relu2", the square of relu) on the columns ``[cols[0], cols[1])``
    (in the product's epilogue in bf16)."""
    if not x.is_cuda:
        gemm(x, w, out=out, bias=bias)
        if cols is not None:
            part = out[:, cols[0]:cols[1]]
            part.copy_(torch.relu(part) ** 2 if act == "relu2" else torch.nn.functional.silu(part))
        return out
    if cols is None or x.dtype == torch.bfloat16:
        return gemm(x, w, out=out, bias=bias, col_act=None if cols is None else (act, *cols))
    gemm(x, w, out=out, bias=bias)
    part = out[:, cols[0]:cols[1]]
    _native.call("tw_act_cols", part.data_ptr(), _row_stride(part), part.shape[0], part.shape[1], COL_ACTS[act], _dt(part),
                 _stream())
    return out


GLU_ACTS = {"silu": 1, "gelu_tanh": 2, "clamped": 3}


def glu(z: torch.Tensor, act: "str | tuple", out: torch.Tensor) -> None:
    """``out = act(z_gate) * z_up`` of rows ``z`` = [gate | up] (CUDA); ``act`` as for :func:`ops.gemm`."""
    kind, limit, alpha = (act, 0.0, 0.0) if isinstance(act, str) else act
    _native.call("tw_glu", z.data_ptr(), _row_stride(z), out.data_ptr(), _row_stride(out), z.shape[0], out.shape[1],
                 GLU_ACTS[kind], float(limit), float(alpha), _dt(z, out), _stream())


def gated_product(x: torch.Tensor, w: torch.Tensor, act: "str | tuple", out: torch.Tensor,
                  tmp: Optional[torch.Tensor]) -> None:
    """``out = act(x w_gate^T) * (x w_up^T)`` with ``w`` = [gate; up] (``act`` as for :func:`ops.gemm`): one product in bf16,
    in fp32 a product into ``tmp`` and the gate behind it."""
    if not x.is_cuda:
        ref.gated_product(x, w, act, out)
        return
    if x.dtype == torch.bfloat16:
        gemm(x, w, out=out, swiglu=True, act=act)
        return
    gemm(x, w, out=tmp)
    glu(tmp, act, out)


# ---- grouped attention ------------------------------------------------------------------------------------------------
QK_NORMS = {None: 0, "head": 1, "whole": 2, "unit": 1}       # "unit": per head, without weights


def qkv_prep(p: torch.Tensor, heads: int, kv_heads: int, dim: int, vdim: int, q: torch.Tensor,
             k_cache: Optional[torch.Tensor], v_cache: Optional[torch.Tensor], meta, conv_w: Optional[torch.Tensor], conv_state: Optional[torch.Tensor],
             qk_norm: Optional[str], wq: Optional[torch.Tensor], wk: Optional[torch.Tensor], eps: float, temp_coef: float,
             temp_every: int, cos_sin: Optional[torch.Tensor] = None) -> None:
    """Everything between the projection and the attention. ``p`` rows are [queries | keys | values], heads padded to
    the caches' last dimension; ``conv_w`` [taps, columns] and ``conv_state`` [slots, taps - 1, columns]: causal
    convolution over time, the state moved on; norm of queries and keys per head (with weights, or "unit") or whole; rotation of the first
    ``cos_sin.shape[1]`` dimensions of every query and key head (dimensions 2i and 2i + 1 are a pair; the table's rows are
    cosines, then sines, by position); queries times ``1 + temp_coef * ln(floor((position + 1) / temp_every) + 1)``; ``q`` [T, heads * padded], keys and values into the
    caches [blocks, page, kv_heads, padded]. Without key heads (and caches) the rows hold queries only."""
    if not p.is_cuda:
        ref.qkv_prep(p, heads, kv_heads, dim, vdim, q, k_cache, v_cache, meta, conv_w, conv_state, qk_norm, wq, wk, eps,
                     temp_coef, temp_every, cos_sin)
        return
    e = meta.extra
    assert cos_sin is None or (cos_sin.dtype == torch.float32 and cos_sin.is_contiguous())
    dp = q.shape[1] // heads
    assert kv_heads == 0 or k_cache.shape[-1] == dp
    _native.call("tw_qkv_prep", p.data_ptr(), _row_stride(p), p.shape[0], heads, kv_heads, dim, dp,
                 v_cache.shape[-1] if v_cache is not None else dp, q.data_ptr(), _row_stride(q), _p(k_cache), _p(v_cache),
                 meta.positions.data_ptr(), meta.slot_mapping.data_ptr(), _p(conv_w), _p(conv_state),
                 conv_w.shape[0] if conv_w is not None else 1, _p(e.get("row_seq")), meta.cu_q.data_ptr(),
                 meta.kv_lens.data_ptr(), _p(e.get("state_slots")), meta.num_seqs, int(meta.all_single),
                 QK_NORMS[qk_norm], _p(wq), _p(wk), float(eps), float(temp_coef), int(temp_every), _p(cos_sin),
                 cos_sin.shape[1] if cos_sin is not None else 0,
                 _dt(p, q, k_cache, v_cache, conv_w, conv_state, wq, wk), _stream())


def attention_tileable(dtype: torch.dtype, dp: int, vp: int) -> bool:
    """Padded head sizes the query-tile kernel takes (bf16)."""
    return dtype == torch.bfloat16 and dp <= 128 and vp <= 128


def attention_rows_plan(n: int, heads: int, kv_heads: int, dp: int, vp: int, page: int, dtype: torch.dtype,
                        max_kv_len: int, sm_count: int = 148, window: int = 0, keep: int = 0) -> tuple[str, int]:
    """(kernel, key splits) for rows attended alone: "tc" (tensor cores) or "simt" (fp32, heads beyond 128 elements)."""
    if dtype != torch.bfloat16 or dp > 128 or vp > 128 or page < 8 or page > 128 or 128 % page:
        return "simt", 1
    blocks = kv_heads * ((heads // kv_heads + 15) // 16)
    return "tc", decode_splits_tc(n * blocks, _key_tiles(max_kv_len, window, keep), sm_count)


def grouped_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, meta, heads: int,
                      kv_heads: int, scale: float, slopes: Optional[torch.Tensor], sink: bool, out_scale: float,
                      sm_count: int = 148, kernel: Optional[str] = None, window: int = 0, keep: int = 0,
                      key_bias: Optional[torch.Tensor] = None, chunk: int = 0, gate: Optional[torch.Tensor] = None) -> None:
    """Causal attention of a step's rows over the paged caches; head h's score loses ``slopes[h] * (i - j)``; ``sink``
    adds one to the denominator; the result is multiplied by ``out_scale``; ``window`` > 0: a row sees the last ``window``
    keys, itself among them, and the sequence's first ``keep``. With ``key_bias`` (fp32 [heads]) there is no softmax: a key
    counts with the sigmoid of its score + ``key_bias[h]``; ``chunk`` > 0: a row sees the keys of its own chunk of that many
    positions, counted from the sequence's start; ``gate`` [T, >= heads]: head h's result times ``sigmoid(gate[:, h])``
    (these options go together, without those of the softmax). ``kernel``: force "simt" (tests)."""
    if key_bias is None and (chunk or gate is not None) or key_bias is not None and (window or sink or slopes is not None):
        raise ValueError("chunks and gates go with sigmoid weights; windows, sinks and distance biases with a softmax")
    if not q.is_cuda:
        ref.grouped_attention(q, k_cache, v_cache, out, meta, heads, kv_heads, scale, slopes, sink, out_scale, window, keep,
                              key_bias, chunk, gate)
        return
    dt = _dt(q, k_cache, v_cache, out, gate)
    assert key_bias is None or key_bias.dtype == torch.float32
    sigmoid = (_p(key_bias), int(chunk), _p(gate), _row_stride(gate) if gate is not None else 0)
    page, dp, vp = k_cache.shape[1], k_cache.shape[-1], v_cache.shape[-1]
    if meta.num_tiles:
        _native.call("tw_attn_prefill_grouped", q.data_ptr(), _row_stride(q), q.shape[0], k_cache.data_ptr(),
                     v_cache.data_ptr(), k_cache.shape[0], page, out.data_ptr(), _row_stride(out), meta.cu_q.data_ptr(),
                     meta.kv_lens.data_ptr(), meta.block_table.data_ptr(), meta.block_table.shape[1],
                     meta.tile_seq.data_ptr(), meta.tile_q0.data_ptr(), meta.num_tiles, heads, kv_heads, dp, vp,
                     float(scale), _p(slopes), int(sink), float(out_scale), int(window), int(keep), *sigmoid,
                     status_word(q.device).data_ptr(), _stream())
    n = meta.num_single
    if n == 0:
        return
    plan, splits = attention_rows_plan(n, heads, kv_heads, dp, vp, page, q.dtype, meta.max_kv_len, sm_count, window or chunk,
                                       keep)
    if (kernel or plan) == "simt":
        _native.call("tw_attn_rows", q.data_ptr(), _row_stride(q), k_cache.data_ptr(), v_cache.data_ptr(), page,
                     out.data_ptr(), _row_stride(out), meta.tok_row.data_ptr(), meta.tok_seq.data_ptr(),
                     meta.tok_kvlen.data_ptr(), n, meta.block_table.data_ptr(), meta.block_table.shape[1], heads, kv_heads,
                     dp, vp, float(scale), _p(slopes), int(sink), float(out_scale), int(window), int(keep), *sigmoid, dt,
                     _stream())
        return
    po = pm = None
    if splits > 1:
        po, pm = _partial_buffers(q.device, n * heads * splits, vp)
    _native.call("tw_attn_decode_grouped", q.data_ptr(), _row_stride(q), k_cache.data_ptr(), v_cache.data_ptr(),
                 k_cache.shape[0], page, out.data_ptr(), _row_stride(out), meta.tok_row.data_ptr(), meta.tok_seq.data_ptr(),
                 meta.tok_kvlen.data_ptr(), n, meta.block_table.data_ptr(), meta.block_table.shape[1], heads, kv_heads, dp,
                 vp, float(scale), _p(slopes), int(sink), float(out_scale), int(window), int(keep), *sigmoid, splits, _p(po),
                 _p(pm),
                 status_word(q.device).data_ptr(), _stream())

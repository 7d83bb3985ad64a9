"""Plain PyTorch implementations of the operators of :mod:`tokenweave_b200.ops.hybrid`: the engine's CPU path (fp32
runs without a GPU) and the per-operator oracle of the kernels. fp32 arithmetic, rounded where the kernels store."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F

from .reference import gemm_clamped


def _unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def embed_residual(ids, table, x32, xa, width: int) -> None:
    ok = (ids >= 0) & (ids < table.shape[0])
    rows = table.index_select(0, torch.where(ok, ids, torch.zeros_like(ids)).long())[:, :width]
    rows = rows * ok.unsqueeze(-1).to(rows.dtype)
    x32[:, :width] = rows.float()
    xa[:, :width] = rows


def postnorm_add_(y, x32, weight, eps: float, xa, final_weight: Optional[torch.Tensor] = None) -> None:
    h = weight.numel()
    x32[:, :h] += _unit(y[:, :h].float(), eps) * weight.float()
    x = x32[:, :h]
    xa[:, :h] = x if final_weight is None else _unit(x, eps) * final_weight.float()


def polynorm(z, coef, eps: float):
    a, b, c, e = coef.float().tolist()
    zf = z.float()
    return (a * _unit(zf, eps) + b * _unit(zf ** 2, eps) + c * _unit(zf ** 3, eps) + e).to(z.dtype)


def gated_group_norm(y, z, weight, groups: int, eps: float):
    v = y.float() * F.silu(z.float())
    v = _unit(v.reshape(v.shape[0], groups, -1), eps).reshape(v.shape)
    return (v * weight.float()).to(y.dtype)


def _rotate(x, cos_sin, positions, rot_dims: int):
    """``x`` [T, ..., rot]: the first rot_dims dimensions rotated in half-split pairs."""
    half = rot_dims // 2
    cs = cos_sin.index_select(0, positions.long())
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    cos, sin = cs[:, :half].reshape(shape), cs[:, half:].reshape(shape)
    u, v = x[..., :half], x[..., half:rot_dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., rot_dims:]], -1)


def _rotate_pairs(x, cos_sin, positions):
    """``x`` [T, heads, D]: the first ``cos_sin.shape[1]`` dimensions rotated, dimensions 2i and 2i + 1 as a pair."""
    dims = cos_sin.shape[1]
    cs = cos_sin.index_select(0, positions.long()).unsqueeze(1)
    cos, sin = cs[..., :dims // 2], cs[..., dims // 2:]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], -1)


def latent_prep(p, q_off, q_rank, wq, cq, kv_off, kv_rank, wkv, rot, rot_dims, cos_sin, positions, slots, cache,
                eps: float) -> None:
    pf = p.float()
    cq[:, :q_rank] = (_unit(pf[:, q_off:q_off + q_rank], eps) * wq.float()).to(cq.dtype)
    row = torch.zeros(p.shape[0], cache.shape[-1], dtype=torch.float32)
    row[:, :kv_rank] = _unit(pf[:, kv_off:kv_off + kv_rank], eps) * wkv.float()
    rp = (kv_rank + 7) // 8 * 8
    kr = pf[:, kv_off + kv_rank:kv_off + kv_rank + rot]
    row[:, rp:rp + rot] = _rotate(kr, cos_sin, positions, rot_dims)
    ok = slots >= 0
    cache.view(-1, cache.shape[-1])[slots[ok].long()] = row[ok].to(cache.dtype)


def latent_absorb(q, rows, w_ukt, heads, dim, rot, rot_dims, kv_rank, cos_sin, positions, row):
    r = rows.long()
    qh = q.index_select(0, r)[:, : heads * (dim + rot)].reshape(-1, heads, dim + rot).float()
    out = torch.zeros(qh.shape[0], heads, row)
    out[..., :kv_rank] = torch.einsum("thd,hrd->thr", qh[..., :dim], w_ukt[..., :dim].float())
    rp = (kv_rank + 7) // 8 * 8
    out[..., rp:rp + rot] = _rotate(qh[..., dim:], cos_sin, positions.index_select(0, r), rot_dims)
    return out.to(q.dtype)


def latent_attention(qa, cache, tok_seq, tok_kvlen, block_table, kv_rank, scale, window: int = 0, sink=None):
    n, heads, _ = qa.shape
    page = cache.shape[1]
    out = torch.empty(n, heads, kv_rank, dtype=qa.dtype)
    seqs, lens = tok_seq.tolist(), tok_kvlen.tolist()
    flat = {}
    for s in set(seqs[:n]):
        top = max(k for i, k in enumerate(lens[:n]) if seqs[i] == s)
        blocks = block_table[s, : (top + page - 1) // page].long()
        flat[s] = cache.index_select(0, blocks).reshape(-1, cache.shape[-1]).float()
    for i in range(n):
        keys = flat[seqs[i]][max(0, lens[i] - window) if window else 0: lens[i]]
        s = qa[i].float() @ keys.t() * scale
        w = torch.softmax(s if sink is None else torch.cat([s, sink[:, None]], -1), -1)[:, :keys.shape[0]]
        out[i] = (w @ keys[:, :kv_rank]).to(qa.dtype)
    return out


def latent_values(o, rows, w_uv, heads, vdim, kv_rank, gate, out) -> None:
    v = torch.einsum("thr,hvr->thv", o.float(), w_uv[..., :kv_rank].float()).reshape(o.shape[0], heads * vdim)
    r = rows.long()
    if gate is not None:
        v = v * torch.sigmoid(gate.index_select(0, r)[:, : heads * vdim].float())
    out[r, : heads * vdim] = v.to(out.dtype)


def _with_past(rows, state, slot: int, past: bool, taps: int):
    """``rows`` behind the taps - 1 inputs before them, and the inputs to keep."""
    before = state[slot].float() if past and taps > 1 else torch.zeros(taps - 1, rows.shape[1])
    full = torch.cat([before, rows], 0)
    return full, full[full.shape[0] - (taps - 1):]


def causal_conv(x, weight, bias, state, out, cu_q, kv_lens, slots) -> None:
    taps, channels = weight.shape
    cu, kv, sl = cu_q.tolist(), kv_lens.tolist(), slots.tolist()
    w = weight.float()
    for b in range(len(kv)):
        rows = x[cu[b]:cu[b + 1], :channels].float()
        full, keep = _with_past(rows, state, sl[b], kv[b] > rows.shape[0], taps)
        y = bias.float() + sum(w[k] * full[k:k + rows.shape[0]] for k in range(taps))
        out[cu[b]:cu[b + 1], :channels] = F.silu(y).to(out.dtype)
        if taps > 1:
            state[sl[b]] = keep.to(state.dtype)


def _recurrence(x, B, C, decay, step, D, state, y, seqs, cu_q, kv_lens, slots) -> None:
    """``S <- decay_t S + step_t x B^T``, ``y = S C + D x``; x [T, H, P], B and C [T, H, N], decay and step [T, H]."""
    cu, kv, sl = cu_q.tolist(), kv_lens.tolist(), slots.tolist()
    _, heads, vdim, N = state.shape
    for b in seqs.tolist():
        s = state[sl[b]].clone() if kv[b] > cu[b + 1] - cu[b] else torch.zeros(heads, vdim, N)
        for t in range(cu[b], cu[b + 1]):
            s = decay[t][:, None, None] * s + (step[t][:, None] * x[t])[:, :, None] * B[t][:, None, :]
            o = torch.einsum("hpn,hn->hp", s, C[t])
            y[t, :heads * vdim] = (o if D is None else o + D[:, None] * x[t]).reshape(-1).to(y.dtype)
        state[sl[b]] = s


def ssd_scan(xbc, dt, dt_bias, A_log, D, state, y, seqs, cu_q, kv_lens, slots, groups: int) -> None:
    _, heads, vdim, N = state.shape
    inner, rep, T = heads * vdim, heads // groups, xbc.shape[0]
    step = F.softplus(dt[:, :heads].float() + dt_bias.float(), threshold=1e9)
    decay = torch.exp(-torch.exp(A_log.float()) * step)
    r = xbc.float()
    B, C = (r[:, inner + i * groups * N:inner + (i + 1) * groups * N].reshape(T, groups, N).repeat_interleave(rep, 1)
            for i in (0, 1))
    _recurrence(r[:, :inner].reshape(T, heads, vdim), B, C, decay, step, D.float(), state, y, seqs, cu_q, kv_lens, slots)


def decay_scan(p, decay, state, y, seqs, cu_q, kv_lens, slots) -> None:
    _, heads, vdim, N = state.shape
    inner, T, r = heads * vdim, p.shape[0], p.float()
    k, q = (r[:, inner + i * heads * N:inner + (i + 1) * heads * N].reshape(T, heads, N) for i in (0, 1))
    one = torch.ones(T, heads)
    _recurrence(r[:, :inner].reshape(T, heads, vdim), k, q, one * decay, one, None, state, y, seqs, cu_q, kv_lens, slots)


# ---- norms on both sides of a sublayer, averages over the depth -----------------------------------------------------
def _norm(x, norm, eps: float):
    w, b = norm
    if b is None:
        return _unit(x, eps) * w.float()
    return _unit(x - x.mean(-1, keepdim=True), eps) * w.float() + b.float()


def embed_sandwich(ids, table, scale: float, x32, first, norm, eps: float, xa) -> None:
    h = norm[0].numel()
    ok = (ids >= 0) & (ids < table.shape[0])
    x = table.index_select(0, torch.where(ok, ids, torch.zeros_like(ids)).long())[:, :h].float() * ok.unsqueeze(-1) * scale
    x32[:, :h] = x
    if first is not None:
        first[:, :h] = x
    xa[:, :h] = _norm(x, norm, eps)


def sandwich_step(y, x32, post, nxt, eps: float, xa, coef, results, last: bool) -> None:
    h = post[0].numel()
    x = x32[:, :h] + _norm(y[:, :h].float(), post, eps)
    if coef is not None:
        n = coef.numel() - 1
        if not last:
            results[n, :, :h] = x
        x = coef[n] * x
        for j in range(n):
            x = x + coef[j] * results[j, :, :h]
    x32[:, :h] = x
    xa[:, :h] = _norm(x, nxt, eps)


def min_gru(p, bz, bx, state, out, seqs, cu_q, kv_lens, slots) -> None:
    n, r = state.shape[1], p.float()
    z, u, g = torch.sigmoid(r[:, :n] + bz), r[:, n:2 * n] + bx, F.silu(r[:, 2 * n:3 * n])
    add = z * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    cu, kv, sl = cu_q.tolist(), kv_lens.tolist(), slots.tolist()
    for b in seqs.tolist():
        s = state[sl[b]].clone() if kv[b] > cu[b + 1] - cu[b] else torch.zeros(n)
        for t in range(cu[b], cu[b + 1]):
            s = (1 - z[t]) * s + add[t]
            out[t, :n] = (s * g[t]).to(out.dtype)
        state[sl[b]] = s


# ---- hyper-connections -------------------------------------------------------------------------------------------
def embed_streams(ids, table, x, hc_in, weight, offset: float, eps: float, xa) -> None:
    h = weight.numel()
    ok = (ids >= 0) & (ids < table.shape[0])
    rows = table.index_select(0, torch.where(ok, ids, torch.zeros_like(ids)).long())[:, :h].float() * ok.unsqueeze(-1)
    x[:, 0, :h] = rows
    xa[:, :h] = _unit(rows * hc_in.sum(), eps) * (offset + weight.float())


def streams_step(y, x, hc, mult: float, next_in, weight, offset: float, eps: float, xa, first: bool = False) -> None:
    h = weight.numel()
    old = x[:, :1, :h].expand(-1, x.shape[1], -1) if first else x[:, :, :h]
    new = torch.einsum("nsw,st->ntw", old, hc["mix"]) + mult * hc["out"][:, None] * y[:, None, :h].float()
    if next_in is None:
        u = new.sum(1)
    else:
        x[:, :, :h] = new
        u = torch.einsum("nsw,s->nw", new, next_in)
    xa[:, :h] = _unit(u, eps) * (offset + weight.float())


# ---- blocks whose sublayers read one norm of the stream ---------------------------------------------------------
def pair_rows(ids, row_seq, cu_q, prev_token, spec):
    """Row of the pair table for every token; its last row for a token without one before it."""
    ids = ids.long()
    prev = torch.cat([ids[:1], ids[:-1]])
    first = cu_q.long()[row_seq.long()] == torch.arange(len(ids))
    prev = torch.where(first, prev_token.long()[row_seq.long()], prev)
    buckets = int(spec["buckets"])
    rows = (prev * int(spec["mul_prev"]) + ids * int(spec["mul_cur"])) % buckets
    return torch.where(prev < 0, torch.full_like(rows, buckets), rows)


def embed_norm(ids, table, pairs, spec, meta, x32, first, weight, eps: float, xa) -> None:
    h = weight.numel()
    ok = (ids >= 0) & (ids < table.shape[0])
    x = table.index_select(0, torch.where(ok, ids, torch.zeros_like(ids)).long())[:, :h].float()
    x = x * ok.unsqueeze(-1)
    if pairs is not None:
        x = x + pairs.index_select(0, pair_rows(ids, meta.extra["row_seq"], meta.cu_q, meta.extra["prev_token"],
                                                spec))[:, :h].float()
    x32[:, :h] = x
    if first is not None:
        first[:, :h] = x
    xa[:, :h] = _unit(x, eps) * weight.float()


def add_prenorm_(y, x32, first, weight, eps: float, xa) -> None:
    h = weight.numel()
    x = x32[:, :h]
    x += y[:, :h].float()
    if first is not None:
        x += first[:, :h]
    xa[:, :h] = _unit(x, eps) * weight.float()


def gated_product(x, w, act, out) -> None:
    if not isinstance(act, str):
        out.copy_(gemm_clamped(x, w, *act[1:]))
        return
    d = w.shape[0] // 2
    z = x.float() @ w.float().t()
    g = F.silu(z[:, :d]) if act == "silu" else F.gelu(z[:, :d], approximate="tanh")
    out.copy_(g * z[:, d:])


def norm_gate(y, gate, weight, count: int, eps: float, scale: float, out) -> None:
    v = y.float()
    r = torch.rsqrt(v.pow(2).sum(-1, keepdim=True) / count + eps)
    out.copy_(v * r * weight.float() * torch.sigmoid(gate.float()) * scale)


def qkv_prep(p, heads: int, kv_heads: int, dim: int, vdim: int, q, k_cache, v_cache, meta, conv_w, conv_state, qk_norm,
             wq, wk, eps: float, temp_coef: float, temp_every: int, cos_sin=None) -> None:
    dp, T = q.shape[1] // heads, p.shape[0]
    x = p.float()
    if conv_w is not None:
        taps, w = conv_w.shape[0], conv_w.float()
        cu, kv, sl = meta.cu_q.tolist(), meta.kv_lens.tolist(), meta.extra.get("state_slots", meta.cu_q).tolist()
        mixed = torch.empty_like(x)
        for b in range(len(kv)):
            rows = x[cu[b]:cu[b + 1]]
            full, keep = _with_past(rows, conv_state, sl[b], kv[b] > rows.shape[0], taps)
            mixed[cu[b]:cu[b + 1]] = sum(w[k] * full[k:k + rows.shape[0]] for k in range(taps))
            if taps > 1:
                conv_state[sl[b]] = keep.to(conv_state.dtype)
        x = mixed
    nq, nk = heads * dp, kv_heads * dp
    vp = v_cache.shape[-1] if kv_heads else 0
    qs, ks, vs = x[:, :nq], x[:, nq:nq + nk], x[:, nq + nk:nq + nk + kv_heads * vp]

    def normed(t, weight, n):
        parts = 1 if qk_norm == "whole" else n
        t = t.reshape(T, parts, -1)
        count = dim * n // parts
        t = t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) / count + eps)
        return (t * weight.float() if weight is not None else t).reshape(T, -1)
    if qk_norm:
        qs, ks = normed(qs, wq, heads), normed(ks, wk, kv_heads) if kv_heads else ks
    if cos_sin is not None:
        qs, ks = (_rotate_pairs(t.reshape(T, n, dp), cos_sin, meta.positions).reshape(T, n * dp)
                  for t, n in ((qs, heads), (ks, kv_heads)))
    if temp_coef:
        turn = torch.div(meta.positions.long() + 1, temp_every, rounding_mode="floor")
        qs = qs * (1 + temp_coef * torch.log(turn.float() + 1)).unsqueeze(-1)
    q.copy_(qs)
    if not kv_heads:
        return
    slots = meta.slot_mapping.long()
    ok = slots >= 0
    k_cache.view(-1, nk)[slots[ok]] = ks[ok].to(k_cache.dtype)
    v_cache.view(-1, kv_heads * vp)[slots[ok]] = vs[ok].to(v_cache.dtype)


def grouped_attention(q, k_cache, v_cache, out, meta, heads: int, kv_heads: int, scale: float, slopes, sink: bool,
                      out_scale: float, window: int = 0, keep: int = 0, key_bias=None, chunk: int = 0, gate=None) -> None:
    page, dp, vp, rep = k_cache.shape[1], k_cache.shape[-1], v_cache.shape[-1], heads // kv_heads
    for b, kv_len in enumerate(meta.kv_lens_cpu):
        t0, t1 = meta.cu_q_cpu[b], meta.cu_q_cpu[b + 1]
        blocks = meta.block_table[b, :(kv_len + page - 1) // page].long()
        k = k_cache.index_select(0, blocks).reshape(-1, kv_heads, dp)[:kv_len].float().repeat_interleave(rep, 1)
        v = v_cache.index_select(0, blocks).reshape(-1, kv_heads, vp)[:kv_len].float().repeat_interleave(rep, 1)
        s = torch.einsum("qhd,khd->hqk", q[t0:t1].reshape(t1 - t0, heads, dp).float(), k) * scale
        dist = torch.arange(kv_len - (t1 - t0), kv_len).unsqueeze(-1) - torch.arange(kv_len)
        if slopes is not None:
            s = s - slopes[:, None, None] * dist
        hidden = dist < 0
        if window:
            hidden = hidden | ((dist >= window) & (torch.arange(kv_len) >= keep))
        if chunk:
            hidden = hidden | (torch.arange(kv_len - (t1 - t0), kv_len).unsqueeze(-1) // chunk != torch.arange(kv_len) // chunk)
        if key_bias is not None:
            w = torch.sigmoid(s + key_bias[:, None, None]).masked_fill(hidden, 0.0)
        else:
            s = s.masked_fill(hidden, float("-inf"))
            if sink:
                s = torch.cat([s, torch.zeros(heads, t1 - t0, 1)], -1)
            w = torch.softmax(s, -1)[..., :kv_len]
        o = torch.einsum("hqk,khd->qhd", w, v) * out_scale
        if gate is not None:
            o = o * torch.sigmoid(gate[t0:t1, :heads].float()).unsqueeze(-1)
        out[t0:t1] = o.reshape(t1 - t0, -1).to(out.dtype)

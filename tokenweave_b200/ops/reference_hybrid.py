"""Plain PyTorch implementations of the operators of :mod:`tokenweave_b200.ops.hybrid`: the engine's CPU path (fp32
runs without a GPU) and the per-operator oracle of the kernels. fp32 arithmetic, rounded where the kernels store."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F


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


def latent_attention(qa, cache, tok_seq, tok_kvlen, block_table, kv_rank, scale):
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
        keys = flat[seqs[i]][: lens[i]]
        w = torch.softmax(qa[i].float() @ keys.t() * scale, -1)
        out[i] = (w @ keys[:, :kv_rank]).to(qa.dtype)
    return out


def latent_values(o, rows, w_uv, heads, vdim, kv_rank, gate, out) -> None:
    v = torch.einsum("thr,hvr->thv", o.float(), w_uv[..., :kv_rank].float()).reshape(o.shape[0], heads * vdim)
    r = rows.long()
    if gate is not None:
        v = v * torch.sigmoid(gate.index_select(0, r)[:, : heads * vdim].float())
    out[r, : heads * vdim] = v.to(out.dtype)


def causal_conv(x, weight, bias, state, out, cu_q, kv_lens, slots) -> None:
    taps, channels = weight.shape
    cu, kv, sl = cu_q.tolist(), kv_lens.tolist(), slots.tolist()
    w = weight.float()
    for b in range(len(kv)):
        rows = x[cu[b]:cu[b + 1], :channels].float()
        past = state[sl[b]].float() if kv[b] > rows.shape[0] else torch.zeros(taps - 1, channels)
        full = torch.cat([past, rows], 0)
        y = bias.float() + sum(w[k] * full[k:k + rows.shape[0]] for k in range(taps))
        out[cu[b]:cu[b + 1], :channels] = F.silu(y).to(out.dtype)
        if taps > 1:
            state[sl[b]] = full[full.shape[0] - (taps - 1):].to(state.dtype)


def ssd_scan(xbc, dt, dt_bias, A_log, D, state, y, seqs, cu_q, kv_lens, slots, groups: int) -> None:
    _, heads, vdim, N = state.shape
    cu, kv, sl = cu_q.tolist(), kv_lens.tolist(), slots.tolist()
    inner, rep = heads * vdim, heads // groups
    step = F.softplus(dt[:, :heads].float() + dt_bias.float(), threshold=1e9)
    decay = torch.exp(-torch.exp(A_log.float()) * step)
    for b in seqs.tolist():
        s = state[sl[b]].clone() if kv[b] > cu[b + 1] - cu[b] else torch.zeros(heads, vdim, N)
        for t in range(cu[b], cu[b + 1]):
            r = xbc[t].float()
            x = r[:inner].reshape(heads, vdim)
            B = r[inner:inner + groups * N].reshape(groups, N).repeat_interleave(rep, 0)
            C = r[inner + groups * N:inner + 2 * groups * N].reshape(groups, N).repeat_interleave(rep, 0)
            s = decay[t][:, None, None] * s + (step[t][:, None] * x)[:, :, None] * B[:, None, :]
            y[t, :inner] = (torch.einsum("hpn,hn->hp", s, C) + D.float()[:, None] * x).reshape(-1).to(y.dtype)
        state[sl[b]] = s

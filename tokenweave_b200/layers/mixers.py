"""Token mixers and feed-forwards of hybrid decoders: layers that a model's configuration lists one by one, each with
its own kind and sizes (``models/hybrid.py``).

A mixer owns its weights and maps activation rows to sublayer outputs: ``forward(x, meta, rt, out, kept)``. What it
keeps between steps - pages of a cache (``cache_bytes_per_block`` / ``init_cache``), a slot of recurrent state per
sequence (``state_bytes_per_slot`` / ``init_state``) - is in ``kept``, which the model makes once per RUN of the layer: a
layer that runs several times in a row has one set of weights and one ``kept`` per pass. All sizes and constants are
parameters, so another design can list the same mixers with other values. :data:`MIXERS` and :data:`FEED_FORWARDS` are
the names a configuration may use.

A :class:`SumMixer` adds up several :class:`Part` s that read the same input (and, where a layer's feed-forward reads
that input too, the feed-forward): their input projections are one matrix product, and so are their output projections.

Activations and weights are bf16 or fp32 (the engine's dtype); norms, rotary angles, attention scores and softmax,
decays and recurrent state are fp32 in both.
"""
from __future__ import annotations

import math
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..ops import hybrid as hops
from ..ops import reference
from .attention import AttentionMetadata
from .linear import PaddedLinear, pad8
from .moe import expert_index, max_expert_rows, run_experts


def _vec(n: int, dtype, device, fill: float = 1.0) -> nn.Parameter:
    return nn.Parameter(torch.full((n,), fill, dtype=dtype, device=device), requires_grad=False)


# ---- rotation ---------------------------------------------------------------------------------------------------------
# ``rot`` = {"base", "dims", "scaling": None or YaRN's {"factor", "original", "fast", "slow"}}
def rotation_key(rot: dict) -> tuple:
    return int(rot["dims"]), float(rot["base"]), tuple(sorted((rot.get("scaling") or {}).items()))


def rope_table(rt, rot: dict) -> torch.Tensor:
    """Cosines and sines by position ([positions, dims]: cosines, then sines), one table per kind of rotation in a model."""
    s, key = rot.get("scaling"), rotation_key(rot)
    if key not in rt.rope_tables:
        scaling = None
        if s:
            factor = float(s["factor"])
            scaling = dict(rope_type="yarn", factor=factor, original_max_position_embeddings=float(s["original"]),
                           beta_fast=float(s["fast"]), beta_slow=float(s["slow"]),
                           attention_factor=0.1 * math.log(factor) + 1.0)
        rt.rope_tables[key] = reference.build_cos_sin_cache(key[0], rt.max_positions, key[1], scaling, rt.device)
    return rt.rope_tables[key]


def check_rotation(rot: dict, size: int) -> int:
    dims = int(rot["dims"])
    if dims % 2 or not 0 < dims <= size:
        raise ValueError(f"rotated dimensions {dims} do not fit a part of {size}")
    return dims


def pair_order(dims: int, size: int, to_halves: bool) -> torch.Tensor:
    """Order of a head's ``size`` dimensions, of which the first ``dims`` turn, that changes neighbouring pairs (2i, 2i + 1)
    into pairs of the two halves (i, i + dims / 2), or back. Queries and keys stored in one such order have the same
    products, so a design's pairing is brought to the kernel's once, in the weights."""
    i = torch.arange(dims)
    order = torch.cat([i[0::2], i[1::2]]) if to_halves else i.view(2, -1).t().reshape(-1)
    return torch.cat([order, torch.arange(dims, size)])


class Mixer(nn.Module):
    recurrent = False            # keeps a state slot per sequence

    def cache_bytes_per_block(self, block_size: int) -> int:
        return 0

    def state_bytes_per_slot(self) -> int:
        return 0

    def new_kept(self) -> dict:
        """What one run of the layer keeps between steps, empty; a tree of dicts of tensors."""
        return {}

    def init_cache(self, kept: dict, num_blocks: int, block_size: int) -> None:
        pass

    def init_state(self, kept: dict, num_slots: int) -> None:
        pass

    def bind_runtime(self, rt) -> None:
        """Called once when the runtime exists: constants on the device."""

    def launch_key(self, meta: AttentionMetadata, block_size: int, sm_count: int) -> tuple:
        """What shapes this mixer's launches besides the step's counts."""
        return ()

    def workspaces(self) -> list[tuple[str, int]]:
        """(name, columns) of the runtime buffers a forward pass uses."""
        raise NotImplementedError

    def tensor_targets(self) -> dict:
        """checkpoint name (behind ``<layer>.mix.``) -> (shape, callable taking the tensor)."""
        raise NotImplementedError


class LatentAttention(Mixer):
    """Latent attention: queries from a normed latent of ``q_rank``, keys and values from a normed latent of
    ``kv_rank`` per token plus one rotated key part of ``rot_dim`` shared by all heads; only the latent and the
    rotated part are cached. Optional output gate ``sigmoid(W_g x)``.

    Two forms of the same product. Absorbed: the head's key map is applied to the query and its value map to the
    weighted latent sum, so attention runs over cache rows directly (decoding, short runs). Expanded: the context's
    keys and values are made from the gathered latents with one matrix product and a tile kernel attends (long runs
    of a prompt).

    Options: ``gated``; ``window`` > 0: a position sees the last ``window`` positions, itself among them; ``sink``: a learned
    number per head whose exponential joins the softmax's denominator; ``neighbour_pairs``: dimensions 2i and 2i + 1 turn
    together (else i and i + dims / 2).
    """

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device, gated: bool = True, window: int = 0,
                 sink: bool = False, neighbour_pairs: bool = False):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim = (int(sizes[k]) for k in ("heads", "dim", "rot_dim", "vdim"))
        self.kv_rank, self.q_rank = int(sizes["kv_rank"]), int(sizes["q_rank"])
        self.scale, self.eps, self.width, self.gated = float(sizes["scale"]), eps, width, gated
        self.rot = dict(sizes["rot"])
        self.rot_dims = check_rotation(self.rot, self.rot_dim)
        self.window = int(window)
        # the kernels turn pairs of halves
        self.rot_order = pair_order(self.rot_dims, self.rot_dim, True) if neighbour_pairs else None
        self.sink = (nn.Parameter(torch.zeros(self.heads, dtype=torch.float32, device=device), requires_grad=False)
                     if sink else None)
        H, q8, kv8 = self.heads, pad8(self.q_rank), pad8(self.kv_rank + self.rot_dim)
        # one projection for everything that reads the layer's input: [query latent | kv latent, rotated part | gate]
        self.kv_off, self.gate_off = q8, q8 + kv8
        self.in_proj = PaddedLinear(width, q8 + kv8 + (H * self.vdim if gated else 0), dtype=dtype, device=device)
        self.q_norm_w = _vec(self.q_rank, dtype, device)
        self.kv_norm_w = _vec(self.kv_rank, dtype, device)
        self.uq_proj = PaddedLinear(self.q_rank, H * (self.dim + self.rot_dim), dtype=dtype, device=device)
        # [keys of all heads | values of all heads] from the latent, and the key maps transposed for absorbed queries
        self.ukv_proj = PaddedLinear(self.kv_rank, H * (self.dim + self.vdim), dtype=dtype, device=device)
        self.ukt_w = nn.Parameter(torch.zeros(H, self.kv_rank, pad8(self.dim), dtype=dtype, device=device), requires_grad=False)
        self.o_proj = PaddedLinear(H * self.vdim, width, dtype=dtype, device=device)
        self.row = hops.latent_row(self.kv_rank, self.rot_dim)
        self.cos_sin: Optional[torch.Tensor] = None

    def workspaces(self) -> list[tuple[str, int]]:
        return [("proj", self.in_proj.out_padded), ("latent_q", self.uq_proj.in_padded),
                ("query", self.uq_proj.out_padded), ("mixed", self.o_proj.in_padded),
                ("absorbed", self.heads * self.row), ("latent_out", self.heads * self.kv_rank)]

    def context_workspaces(self) -> list[tuple[str, int]]:
        """Buffers with one row per context token of the expanded form."""
        return [("ctx_latent", self.row), ("ctx_kv", self.ukv_proj.out_padded)]

    @property
    def expandable(self) -> bool:
        w = self.o_proj.weight
        return w.is_cuda and hops.latent_expandable(w.dtype, self.dim, self.rot_dim, self.vdim)

    def launch_key(self, meta: AttentionMetadata, block_size: int, sm_count: int) -> tuple:
        return hops.latent_decode_plan(meta.num_single, self.heads, self.row, self.kv_rank, block_size,
                                       self.o_proj.weight.dtype, meta.max_kv_len, sm_count, self.window)

    # ---- cache -----------------------------------------------------------------------------------------
    def cache_bytes_per_block(self, block_size: int) -> int:
        return block_size * self.row * self.o_proj.weight.element_size()

    def init_cache(self, kept: dict, num_blocks: int, block_size: int) -> None:
        w = self.o_proj.weight
        kept["latents"] = torch.zeros(num_blocks, block_size, self.row, dtype=w.dtype, device=w.device)

    def bind_runtime(self, rt) -> None:
        self.cos_sin = rope_table(rt, self.rot)

    # ---- weights ---------------------------------------------------------------------------------------
    def tensor_targets(self) -> dict:
        H, D, V, R, Q, W = self.heads, self.dim, self.vdim, self.kv_rank, self.q_rank, self.width

        def uk(t):
            self.ukv_proj.load_rows(t, 0)
            self.ukt_w.data[:, :, :D].copy_(t.view(H, D, R).transpose(1, 2))

        def reordered(t, heads, size):
            """Rows of the rotated part, the last of every head's, in the kernels' order of pairs."""
            if self.rot_order is None:
                return t
            order = torch.cat([torch.arange(size - self.rot_dim), size - self.rot_dim + self.rot_order])
            return t.view(heads, size, -1)[:, order.to(t.device)].reshape(t.shape)
        out = {
            "dq": ((Q, W), lambda t: self.in_proj.load_rows(t, 0)),
            "dq.norm": ((Q,), self.q_norm_w.data.copy_),
            "uq": ((H * (D + self.rot_dim), Q), lambda t: self.uq_proj.load_rows(reordered(t, H, D + self.rot_dim), 0)),
            "dkv": ((R + self.rot_dim, W),
                    lambda t: self.in_proj.load_rows(reordered(t, 1, R + self.rot_dim), self.kv_off)),
            "dkv.norm": ((R,), self.kv_norm_w.data.copy_),
            "uk": ((H * D, R), uk),
            "uv": ((H * V, R), lambda t: self.ukv_proj.load_rows(t, H * D)),
            "o": ((W, H * V), lambda t: self.o_proj.load_rows(t, 0)),
        }
        if self.gated:
            out["g"] = ((H * V, W), lambda t: self.in_proj.load_rows(t, self.gate_off))
        if self.sink is not None:
            out["sink"] = ((H,), self.sink.data.copy_)
        return out

    # ---- forward ---------------------------------------------------------------------------------------
    def forward(self, x: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor, kept: dict) -> None:
        n, H, cache = x.shape[0], self.heads, kept["latents"]
        p = self.in_proj(x, out=rt.buffer("proj", n, self.in_proj.out_padded))
        cq = rt.buffer("latent_q", n, self.uq_proj.in_padded)
        hops.latent_prep(p, 0, self.q_rank, self.q_norm_w, cq, self.kv_off, self.kv_rank, self.kv_norm_w, self.rot_dim,
                         self.rot_dims, self.cos_sin, meta.positions, meta.slot_mapping, cache, self.eps)
        q = self.uq_proj(cq, out=rt.buffer("query", n, self.uq_proj.out_padded))
        gate = p[:, self.gate_off:] if self.gated else None
        attn = rt.buffer("mixed", n, self.o_proj.in_padded)
        w_uv = self.ukv_proj.weight[H * self.dim: H * (self.dim + self.vdim)].view(H, self.vdim, -1)
        if meta.num_single:
            m = meta.num_single
            qa = rt.buffer("absorbed", m, H * self.row).view(m, H, self.row)
            hops.latent_absorb(q, meta.tok_row, self.ukt_w, H, self.dim, self.rot_dim, self.rot_dims, self.kv_rank,
                               self.cos_sin, meta.positions, qa)
            o = rt.buffer("latent_out", m, H * self.kv_rank).view(m, H, self.kv_rank)
            hops.latent_attention(qa, cache, meta.tok_seq, meta.tok_kvlen, m, meta.block_table, self.kv_rank,
                                  self.scale, o, meta.max_kv_len, rt.sm_count, window=self.window, sink=self.sink)
            hops.latent_values(o, meta.tok_row, w_uv, H, self.vdim, self.kv_rank, gate, attn)
        if meta.num_tiles:
            # keys and values of the tiles' contexts (the step's own tokens are in the cache already)
            rows = meta.extra_cpu["ctx_rows"]
            lat = rt.buffer("ctx_latent", rows, self.row)
            hops.latent_gather(cache, meta.extra["ctx_seqs"], meta.extra["ctx_cu"], meta.extra_cpu["ctx_max"],
                               meta.block_table, lat, meta.extra["ctx_first"])
            kv = self.ukv_proj(lat[:, :self.ukv_proj.in_padded], out=rt.buffer("ctx_kv", rows, self.ukv_proj.out_padded))
            hops.rope_tail_(q, H, self.dim + self.rot_dim, self.dim, self.rot_dims, self.cos_sin, meta.positions)
            hops.latent_prefill(q, kv, lat, pad8(self.kv_rank), rows, meta.extra["ctx_begin"], attn, gate, meta.cu_q,
                                meta.kv_lens, meta.tile_seq, meta.tile_q0, meta.num_tiles, H, self.dim, self.rot_dim,
                                self.vdim, self.scale, self.window, self.sink)
        self.o_proj(attn, out=out)


class Mamba2Mixer(Mixer):
    """Mamba-2: projection to [gate z | x, B, C | step sizes], causal convolution + silu of x, B and C, state-space
    recurrence per head with an fp32 state, skip ``D x``, gate, grouped RMS norm, output projection."""
    recurrent = True

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device):
        super().__init__()
        self.heads, self.vdim, self.N, self.groups = (int(sizes[k]) for k in ("heads", "vdim", "state", "groups"))
        self.taps, self.norm_groups = int(sizes["conv"]), int(sizes["norm_groups"])
        if self.heads % self.groups:
            raise ValueError(f"{self.heads} heads do not divide into {self.groups} groups")
        self.eps, self.width = eps, width
        self.inner = self.heads * self.vdim
        if self.inner % self.norm_groups:
            raise ValueError(f"{self.inner} channels do not divide into {self.norm_groups} norm groups")
        self.channels = self.inner + 2 * self.groups * self.N
        # every part starts on a 16-byte boundary of the projection's rows
        self.x_off = pad8(self.inner)
        self.dt_off = self.x_off + pad8(self.channels)
        self.in_proj = PaddedLinear(width, self.dt_off + self.heads, dtype=dtype, device=device)
        self.conv_w = nn.Parameter(torch.zeros(self.taps, self.channels, dtype=dtype, device=device), requires_grad=False)
        self.conv_b = _vec(self.channels, dtype, device, 0.0)
        self.dt_bias = _vec(self.heads, dtype, device, 0.0)
        self.A_log = _vec(self.heads, dtype, device, 0.0)
        self.D = _vec(self.heads, dtype, device)
        self.norm_w = _vec(self.inner, dtype, device)
        self.o_proj = PaddedLinear(self.inner, width, dtype=dtype, device=device)

    def workspaces(self) -> list[tuple[str, int]]:
        return [("proj", self.in_proj.out_padded), ("conv", pad8(self.channels)), ("mixed", self.o_proj.in_padded),
                ("gated", self.o_proj.in_padded)]

    @property
    def chunkable(self) -> bool:
        return self.conv_w.is_cuda and hops.ssd_chunkable(self.conv_w.dtype, self.vdim, self.N)

    # ---- state -----------------------------------------------------------------------------------------
    def state_bytes_per_slot(self) -> int:
        return 4 * self.inner * self.N + (self.taps - 1) * self.channels * self.conv_w.element_size()

    def init_state(self, kept: dict, num_slots: int) -> None:
        dev = self.conv_w.device
        kept["state"] = torch.zeros(num_slots, self.heads, self.vdim, self.N, dtype=torch.float32, device=dev)
        kept["conv"] = torch.zeros(num_slots, self.taps - 1, self.channels, dtype=self.conv_w.dtype, device=dev)

    # ---- weights ---------------------------------------------------------------------------------------
    def tensor_targets(self) -> dict:
        I, H, W = self.inner, self.heads, self.width

        def load_in(t):
            z, xbc, dt = t.split([I, self.channels, H], 0)
            self.in_proj.load_rows(z, 0)
            self.in_proj.load_rows(xbc, self.x_off)
            self.in_proj.load_rows(dt, self.dt_off)
        return {
            "in": ((I + self.channels + H, W), load_in),
            "conv": ((self.channels, self.taps), lambda t: self.conv_w.data.copy_(t.t())),
            "conv.b": ((self.channels,), self.conv_b.data.copy_),
            "dt_bias": ((H,), self.dt_bias.data.copy_),
            "A_log": ((H,), self.A_log.data.copy_),
            "D": ((H,), self.D.data.copy_),
            "norm": ((I,), self.norm_w.data.copy_),
            "o": ((W, I), lambda t: self.o_proj.load_rows(t, 0)),
        }

    # ---- forward ---------------------------------------------------------------------------------------
    def forward(self, x: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor, kept: dict) -> None:
        n = x.shape[0]
        p = self.in_proj(x, out=rt.buffer("proj", n, self.in_proj.out_padded))
        xbc = rt.buffer("conv", n, pad8(self.channels))
        e = meta.extra
        hops.causal_conv(p[:, self.x_off:], self.conv_w, self.conv_b, kept["conv"], xbc, e["row_seq"], meta.cu_q,
                         meta.kv_lens, e["state_slots"], meta.all_single)
        y = rt.buffer("mixed", n, self.o_proj.in_padded)
        # long runs in chunks on the tensor cores (sizes permitting), everything else token by token
        for run, seqs in ((hops.ssd_scan, e["scan_seqs"]),
                          (hops.ssd_chunk if self.chunkable else hops.ssd_scan, e["chunk_seqs"])):
            run(xbc, p[:, self.dt_off:], self.dt_bias, self.A_log, self.D, kept["state"], y, seqs, meta.cu_q, meta.kv_lens,
                e["state_slots"], self.groups)
        g = rt.buffer("gated", n, self.o_proj.in_padded)
        hops.gated_group_norm(y, p, self.norm_w, self.norm_groups, self.eps, g)
        self.o_proj(g, out=out)


class MinGRUMixer(Mixer):
    """minGRU: a recurrence per channel whose gates read the current token alone. ``z = sigmoid(W_z x + b_z)``,
    ``u = W_x x + b_x``, ``S <- (1 - z) S + z (u + 1/2 if u >= 0 else sigmoid(u))`` with an fp32 state, output projection of
    ``S silu(W_g x)``. One product makes z, u and the gate; their biases are added in fp32 behind it."""
    recurrent = True

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device):
        super().__init__()
        self.inner, self.width = int(sizes["width"]), width
        self.padded = pad8(self.inner)
        self.in_proj = PaddedLinear(width, 3 * self.padded, dtype=dtype, device=device)
        self.z_bias, self.x_bias = (_vec(self.padded, torch.float32, device, 0.0) for _ in range(2))
        self.o_proj = PaddedLinear(self.inner, width, dtype=dtype, device=device)

    def workspaces(self) -> list[tuple[str, int]]:
        return [("proj", self.in_proj.out_padded), ("mixed", self.o_proj.in_padded)]

    def state_bytes_per_slot(self) -> int:
        return 4 * self.padded

    def init_state(self, kept: dict, num_slots: int) -> None:
        kept["state"] = torch.zeros(num_slots, self.padded, dtype=torch.float32, device=self.z_bias.device)

    def tensor_targets(self) -> dict:
        I, W, P = self.inner, self.width, self.padded
        out = {name: ((I, W), lambda t, row=row: self.in_proj.load_rows(t, row)) for name, row in (("z", 0), ("x", P), ("g", 2 * P))}
        out.update({name: ((I,), b.data[:I].copy_) for name, b in (("z.b", self.z_bias), ("x.b", self.x_bias))})
        out["o"] = ((W, I), lambda t: self.o_proj.load_rows(t, 0))
        return out

    def forward(self, x: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor, kept: dict) -> None:
        n, e = x.shape[0], meta.extra
        p = self.in_proj(x, out=rt.buffer("proj", n, self.in_proj.out_padded))
        y = rt.buffer("mixed", n, self.o_proj.in_padded)
        for seqs, chunked in ((e["scan_seqs"], False), (e["chunk_seqs"], True)):
            hops.min_gru(p, self.z_bias, self.x_bias, kept["state"], y, seqs, meta.cu_q, meta.kv_lens, e["state_slots"], chunked)
        self.o_proj(y, out=out)


class FeedForward(nn.Module):
    """A sublayer without state: ``forward(x, rt, out)``."""

    def workspaces(self) -> list[tuple[str, int]]:
        """(name, columns) of the runtime buffers with a row per token."""
        raise NotImplementedError

    def bind_runtime(self, rt) -> None:
        """Called once when the runtime exists: buffers of other shapes."""

    def tensor_targets(self) -> dict:
        """checkpoint name (behind ``<layer>.mlp.``) -> (shape, callable taking the tensor)."""
        raise NotImplementedError


class PolyNormMLP(FeedForward):
    """``W_down act(W_up x)`` with the polynomial-norm activation ``a N(z) + b N(z^2) + c N(z^3) + e``."""

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device):
        super().__init__()
        self.ff, self.width, self.eps = int(sizes["ff"]), width, eps
        self.up_proj = PaddedLinear(width, self.ff, dtype=dtype, device=device)
        self.down_proj = PaddedLinear(self.ff, width, dtype=dtype, device=device)
        self.coef = _vec(4, dtype, device, 0.0)

    def workspaces(self) -> list[tuple[str, int]]:
        return [("proj", self.up_proj.out_padded), ("act", self.down_proj.in_padded)]

    def tensor_targets(self) -> dict:
        return {"up": ((self.ff, self.width), lambda t: self.up_proj.load_rows(t, 0)),
                "down": ((self.width, self.ff), lambda t: self.down_proj.load_rows(t, 0)),
                "act": ((4,), self.coef.data.copy_)}

    def forward(self, x: torch.Tensor, rt, out: torch.Tensor) -> None:
        n = x.shape[0]
        z = self.up_proj(x, out=rt.buffer("proj", n, self.up_proj.out_padded))
        a = hops.polynorm(z, self.coef, self.eps, rt.buffer("act", n, self.down_proj.in_padded), self.ff)
        self.down_proj(a, out=out)


class ActMLP(FeedForward):
    """``W_down act(W_up x)`` with an elementwise activation: "relu2" (the square of relu) or "silu"."""

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device):
        super().__init__()
        self.ff, self.width, self.act = int(sizes["ff"]), width, str(sizes["act"])
        if self.act not in ops.COL_ACTS:
            raise ValueError(f"unknown activation {self.act!r} (known: {sorted(ops.COL_ACTS)})")
        self.up_proj = PaddedLinear(width, self.ff, dtype=dtype, device=device)
        self.down_proj = PaddedLinear(self.ff, width, dtype=dtype, device=device)

    def workspaces(self) -> list[tuple[str, int]]:
        return [("act", self.down_proj.in_padded)]

    def tensor_targets(self) -> dict:
        return {"up": ((self.ff, self.width), lambda t: self.up_proj.load_rows(t, 0)),
                "down": ((self.width, self.ff), lambda t: self.down_proj.load_rows(t, 0))}

    def forward(self, x: torch.Tensor, rt, out: torch.Tensor) -> None:
        a = rt.buffer("act", x.shape[0], self.down_proj.in_padded)
        hops.projection(x, self.up_proj.weight, None, (0, self.up_proj.out_padded), a, self.act)
        self.down_proj(a, out=out)


class RoutedMLP(FeedForward):
    """Mixture of experts: every token takes ``top`` of ``experts`` gated feed-forwards, chosen by their scores: the softmax
    over all experts, or (``scores`` "sigmoid") each logit's sigmoid; with ``correction`` a number per expert joins the scores
    for the choice. Their weights are the scores (without it), with ``normalize`` over the scores' sum + ``sum_eps``; a weight
    is on the expert's output or (``weigh`` "input") on its input. ``act``: as for ``ops.gemm``. ``shared`` = {"ff", "act",
    "gated"} or None: one more gated feed-forward that every token takes, with "gated" (the default) times the sigmoid of a
    projection to one number.

    The router's rows and the shared feed-forward's gate are one product; the pipeline behind it is ``layers/moe.py``."""

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device):
        super().__init__()
        self.experts, self.top, self.ff, self.width = (*(int(sizes[k]) for k in ("experts", "top", "ff")), width)
        if not 0 < self.top <= self.experts:
            raise ValueError(f"{self.top} of {self.experts} experts")
        self.act, self.sum_eps = self._act(sizes["act"]), float(sizes.get("sum_eps", 0.0))
        self.scores, self.normalize = str(sizes.get("scores", "softmax")), bool(sizes.get("normalize", True))
        if self.scores not in ("softmax", "sigmoid") or sizes.get("weigh", "output") not in ("output", "input"):
            raise ValueError(f"unknown scores {self.scores!r} or place of the weights {sizes.get('weigh')!r}")
        self.weigh_input = sizes.get("weigh") == "input"
        w8, self.f8 = pad8(width), pad8(self.ff)
        par = lambda *s, dt=dtype: nn.Parameter(torch.zeros(*s, dtype=dt, device=device), requires_grad=False)
        shared = sizes.get("shared")
        self.shared_gate = bool(shared) and bool(shared.get("gated", True))
        self.router_w = par(self.experts + int(self.shared_gate), w8)
        self.correction = par(self.experts, dt=torch.float32) if sizes.get("correction", True) else None
        self.w13, self.w2 = par(self.experts, 2 * self.f8, w8), par(self.experts, w8, self.f8)
        self.shared_up = self.shared_down = None
        if shared:
            self.shared_ff, self.shared_act = int(shared["ff"]), self._act(shared["act"])
            self.shared_up = PaddedLinear(width, 2 * pad8(self.shared_ff), dtype=dtype, device=device)
            self.shared_down = PaddedLinear(self.shared_ff, width, dtype=dtype, device=device)

    @staticmethod
    def _act(act):
        return act if isinstance(act, str) else (act[0], float(act[1]), float(act[2]))

    # ---- buffers -------------------------------------------------------------------------------------------
    def workspaces(self) -> list[tuple[str, int]]:
        if self.shared_up is None:
            return []
        out = [("shared_act", self.shared_down.in_padded), ("shared_out", self.shared_down.out_padded)]
        return out + ([("shared_gate_up", self.shared_up.out_padded)] if self.w2.dtype == torch.float32 else [])

    def _sorted_rows(self) -> list[tuple[str, int]]:
        w8 = self.w2.shape[1]
        out = [("a_sorted", w8), ("act", self.f8), ("y", w8)]
        return out + ([("gate_up", 2 * self.f8)] if self.w2.dtype == torch.float32 else [])

    def bind_runtime(self, rt) -> None:
        if not self.w2.is_cuda:
            return
        key = ("experts", self.experts, self.top)
        if key not in rt.tables:
            rt.tables[key] = expert_index(rt.max_tokens, self.top, self.experts, self.w2.device)
        for name, cols in self._sorted_rows():
            rt.buffer("experts." + name, max_expert_rows(rt.max_tokens, self.top, self.experts), cols)

    # ---- weights -------------------------------------------------------------------------------------------
    def tensor_targets(self) -> dict:
        W, F, f8 = self.width, self.ff, self.f8
        out = {"router": ((self.experts, W), lambda t: self.router_w.data[:self.experts, :W].copy_(t))}
        if self.correction is not None:
            out["correction"] = ((self.experts,), self.correction.data.copy_)
        for e in range(self.experts):
            out[f"e{e}.gate"] = ((F, W), lambda t, e=e: self.w13.data[e, :F, :W].copy_(t))
            out[f"e{e}.up"] = ((F, W), lambda t, e=e: self.w13.data[e, f8:f8 + F, :W].copy_(t))
            out[f"e{e}.down"] = ((W, F), lambda t, e=e: self.w2.data[e, :W, :F].copy_(t))
        if self.shared_up is not None:
            S = self.shared_ff
            out["shared.gate"] = ((S, W), lambda t: self.shared_up.load_rows(t, 0))
            out["shared.up"] = ((S, W), lambda t: self.shared_up.load_rows(t, pad8(S)))
            out["shared.down"] = ((W, S), lambda t: self.shared_down.load_rows(t, 0))
        if self.shared_gate:
            out["shared.sg"] = ((1, W), lambda t: self.router_w.data[self.experts:, :W].copy_(t))
        return out

    # ---- forward -------------------------------------------------------------------------------------------
    def forward(self, x: torch.Tensor, rt, out: torch.Tensor) -> None:
        n, shared, gate = x.shape[0], None, None
        weights, ids, gates = ops.moe_route(x, self.router_w, self.experts, self.top, self.correction, self.sum_eps,
                                            self.scores, self.normalize)
        if self.shared_up is not None:
            a = rt.buffer("shared_act", n, self.shared_down.in_padded)
            tmp = rt.buffer("shared_gate_up", n, self.shared_up.out_padded) if x.dtype == torch.float32 else None
            hops.gated_product(x, self.shared_up.weight, self.shared_act, a, tmp)
            shared = self.shared_down(a, out=rt.buffer("shared_out", n, self.shared_down.out_padded))
            gate = gates[:, 0] if self.shared_gate else None
        if not x.is_cuda:
            y = reference.moe_experts(x, self.w13, self.w2, weights, ids, self.act, self.weigh_input)
            out.copy_(y if shared is None else y + (shared if gate is None else gate[:, None] * shared))
            return
        ws = dict(rt.tables[("experts", self.experts, self.top)])
        rows = max_expert_rows(n, self.top, self.experts)
        ws.update((name, rt.buffer("experts." + name, rows, cols)) for name, cols in self._sorted_rows())
        run_experts(x, weights, ids, self.w13, self.w2, ws, out, self.act, shared, gate, weigh_input=self.weigh_input)


# ---- several parts side by side --------------------------------------------------------------------------------------
class Part(nn.Module):
    """One summand of a :class:`SumMixer`. It reads its ``in_cols`` columns of the shared input projection and writes its
    ``out_cols`` columns of the row that the shared output projection takes (both multiples of eight; heads are stored
    padded to eight elements, pads are zero). ``silu_cols``: the projection applies silu to that many of its first
    columns. What it keeps between steps: as for a :class:`Mixer`."""
    in_cols = out_cols = silu_cols = 0
    biased = False               # its projections have biases
    recurrent = False
    attends = False              # attention over cached keys: rows are routed to query tiles or single rows

    cache_bytes_per_block = Mixer.cache_bytes_per_block
    state_bytes_per_slot = Mixer.state_bytes_per_slot
    init_cache, init_state, bind_runtime, launch_key = (Mixer.init_cache, Mixer.init_state, Mixer.bind_runtime,
                                                        Mixer.launch_key)
    tileable = False             # long runs may go to 128-query tiles

    def workspaces(self) -> list[tuple[str, int]]:
        return []

    def tensor_targets(self, width: int, load_in, load_bias, load_out) -> dict:
        """checkpoint name -> (shape, callable). ``load_in(t, row)`` / ``load_bias(t, row)`` / ``load_out(t, col)`` write
        into the shared projections, counted from this part's first row or column."""
        raise NotImplementedError

    def mix(self, p: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor, kept: dict) -> None:
        raise NotImplementedError


def _by_head(load, dim: int, padded: int, base: int):
    """Spreads the rows of ``t`` (heads of ``dim``) over heads of ``padded`` rows from ``base`` on."""
    def put(t: torch.Tensor) -> None:
        for h in range(t.shape[0] // dim):
            load(t[h * dim:(h + 1) * dim], base + h * padded)
    return put


def _pad_heads(dst: torch.Tensor, heads: int, dim: int, padded: int):
    """Writes a vector of ``heads * dim`` elements into ``dst`` [..., heads * padded] (last axis)."""
    def put(t: torch.Tensor) -> None:
        dst.data.view(*dst.shape[:-1], heads, padded)[..., :dim].copy_(t.reshape(*dst.shape[:-1], heads, dim))
    return put


class GroupedAttention(Part):
    """Grouped-query attention with its own sizes of queries / keys (``dim``) and values (``vdim``) over a paged cache.
    Options, each a parameter:

    * ``bias``: biases of the three projections;
    * ``conv``: a causal convolution of that many taps over time on every channel of q, k and v, right behind the
      projection (no bias, no activation); the last ``conv - 1`` projected rows of a sequence are part of its state;
    * ``qk_norm``: "head" (RMS norm of every query and key head, one weight for all), "unit" (the same without a weight),
      "whole" (RMS norm of all queries, and of all keys, of a token at once) or None;
    * ``q_temp`` = {"coef", "every"}: queries times ``1 + coef * ln(floor((p + 1) / every) + 1)`` at position p;
    * ``distance_bias``: ``2^(-8 (h + 1) / heads) * (i - j)`` is taken off the score of head h;
    * ``sink``: one is added to the softmax's denominator (a key of score 0 without a value);
    * ``out_scale``: factor on the result;
    * ``rot``: rotation of the first ``rot["dims"]`` dimensions of queries and keys, behind the norm;
      ``neighbour_pairs``: dimensions 2i and 2i + 1 turn together (else i and i + dims / 2);
    * ``window`` > 0: a position sees the last ``window`` positions, itself among them, and the sequence's first
      ``keep_first``;
    * ``weights``: "softmax", or "sigmoid": a key counts with the sigmoid of its score plus a learned number per head, and
      nothing is normalized (no sink, window or distance bias then); with it ``chunk`` > 0: a position sees the positions of
      its own chunk of that many, counted from the sequence's start; ``head_gate``: each head's result times the sigmoid of a
      projection of the input to one number per head;
    * ``kv_from``: the layer whose keys and values this one reads, as that layer's cache holds them: no projections and no
      cache of its own for them.
    """
    attends = True

    def __init__(self, sizes: dict, eps: float, *, dtype, device, bias: bool = False, conv: Optional[int] = None,
                 qk_norm: Optional[str] = None, q_temp: Optional[dict] = None, distance_bias: bool = False,
                 sink: bool = False, out_scale: float = 1.0, rot: Optional[dict] = None, neighbour_pairs: bool = False,
                 window: int = 0, keep_first: int = 0, weights: str = "softmax", chunk: int = 0, head_gate: bool = False,
                 kv_from: Optional[int] = None):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = (int(sizes[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not divide into {self.kv_heads} groups")
        if qk_norm not in hops.QK_NORMS:
            raise ValueError(f"unknown query and key norm {qk_norm!r}")
        if weights not in ("softmax", "sigmoid"):
            raise ValueError(f"unknown attention weights {weights!r}")
        if (window or sink or distance_bias) if weights == "sigmoid" else (chunk or head_gate):
            raise ValueError("chunks and head gates go with sigmoid weights; windows, sinks and distance biases with a softmax")
        if kv_from is not None and (conv or bias):
            raise ValueError("a layer that reads another's keys and values has no convolution or biases of its own")
        self.scale, self.eps, self.dtype, self.taps = float(sizes["scale"]), eps, dtype, int(conv or 0)
        self.qk_norm, self.distance_bias, self.sink, self.out_scale = qk_norm, distance_bias, sink, float(out_scale)
        self.temp_coef, self.temp_every = (float(q_temp["coef"]), int(q_temp["every"])) if q_temp else (0.0, 1)
        self.biased, self.recurrent = bias, self.taps > 1
        self.dp, self.vp = pad8(self.dim), pad8(self.vdim)
        self.k_off = self.heads * self.dp
        self.kv_from = kv_from
        self.own_kv = 0 if kv_from is not None else self.kv_heads        # key heads that it projects and keeps
        self.v_off = self.k_off + self.own_kv * self.dp
        self.g_off = self.v_off + self.own_kv * self.vp
        self.in_cols, self.out_cols = self.g_off + (pad8(self.heads) if head_gate else 0), self.heads * self.vp
        self.chunk, self.head_gate = int(chunk), head_gate
        self.key_bias = (nn.Parameter(torch.zeros(self.heads, dtype=torch.float32, device=device), requires_grad=False)
                         if weights == "sigmoid" else None)
        self.conv_w = self.q_norm_w = self.k_norm_w = None
        if self.taps:
            self.conv_w = nn.Parameter(torch.zeros(self.taps, self.in_cols, dtype=dtype, device=device), requires_grad=False)
        if qk_norm in ("head", "whole"):
            n = (1, 1) if qk_norm == "head" else (self.heads, self.kv_heads)
            self.q_norm_w, self.k_norm_w = (_vec(i * self.dp, dtype, device, 0.0) for i in n)
        self.device = torch.device(device)
        self.slopes: Optional[torch.Tensor] = None
        self.rot, self.window, self.keep = (dict(rot) if rot else None), int(window), int(keep_first)
        # the kernels turn neighbouring pairs
        self.rot_order = (pair_order(check_rotation(rot, self.dim), self.dim, False)
                          if rot and not neighbour_pairs else None)
        if rot:
            check_rotation(rot, self.dim)
        self.cos_sin: Optional[torch.Tensor] = None

    def bind_runtime(self, rt) -> None:
        if self.rot:
            self.cos_sin = rope_table(rt, self.rot)
        if self.distance_bias:
            h = torch.arange(1, self.heads + 1, dtype=torch.float64)
            self.slopes = torch.exp2(-8.0 * h / self.heads).float().to(self.device)

    def workspaces(self) -> list[tuple[str, int]]:
        return [("query", self.k_off)]

    # ---- cache and state ---------------------------------------------------------------------------------
    def cache_bytes_per_block(self, block_size: int) -> int:
        return block_size * self.own_kv * (self.dp + self.vp) * self.dtype.itemsize

    def init_cache(self, kept: dict, num_blocks: int, block_size: int) -> None:
        if self.kv_from is not None:
            return                           # :meth:`SumMixer.share_cache`
        for name, n in (("k", self.dp), ("v", self.vp)):
            kept[name] = torch.zeros(num_blocks, block_size, self.kv_heads, n, dtype=self.dtype, device=self.device)

    def reads(self, other: "GroupedAttention") -> bool:
        """Whether ``other``'s cache holds keys and values as this part would have made them."""
        alike = lambda p: (p.kv_heads, p.dim, p.vdim, p.dtype, p.rot and rotation_key(p.rot), p.rot_order is None)
        return isinstance(other, GroupedAttention) and other.kv_from is None and alike(self) == alike(other)

    def state_bytes_per_slot(self) -> int:
        return max(0, self.taps - 1) * self.in_cols * self.dtype.itemsize

    def init_state(self, kept: dict, num_slots: int) -> None:
        if self.taps > 1:
            kept["conv"] = torch.zeros(num_slots, self.taps - 1, self.in_cols, dtype=self.dtype, device=self.device)

    # ---- launches ------------------------------------------------------------------------------------------
    @property
    def tileable(self) -> bool:
        return (self.device.type == "cuda" and hops.attention_tileable(self.dtype, self.dp, self.vp)
                and not (self.window and self.distance_bias))

    def launch_key(self, meta: AttentionMetadata, block_size: int, sm_count: int) -> tuple:
        return hops.attention_rows_plan(meta.num_single, self.heads, self.kv_heads, self.dp, self.vp, block_size, self.dtype,
                                        meta.max_kv_len, sm_count, self.window or self.chunk, self.keep)

    # ---- weights -------------------------------------------------------------------------------------------
    def _reordered(self, t: torch.Tensor) -> torch.Tensor:
        """Something with a leading axis of query or key dimensions, in the kernels' order of pairs."""
        if self.rot_order is None:
            return t
        return t.reshape(-1, self.dim, *t.shape[1:])[:, self.rot_order.to(t.device)].reshape(t.shape)

    def tensor_targets(self, width: int, load_in, load_bias, load_out) -> dict:
        H, G, D, V = self.heads, self.kv_heads, self.dim, self.vdim
        spans = {"q": (H, D, self.dp, 0)}
        if self.kv_from is None:
            spans.update(k=(G, D, self.dp, self.k_off), v=(G, V, self.vp, self.v_off))
        out = {"o": ((width, H * V), lambda t: _by_head(lambda r, i: load_out(r.t(), i), V, self.vp, 0)(t.t()))}
        for name, (n, d, padded, base) in spans.items():
            out[name] = ((n * d, width), _by_head(load_in, d, padded, base))
            if self.biased:
                out[name + ".b"] = ((n * d,), _by_head(load_bias, d, padded, base))
            if self.taps:
                put = _pad_heads(self.conv_w[:, base:base + n * padded], n, d, padded)
                out[name + ".conv"] = ((n * d, self.taps), lambda t, put=put: put(t.t()))
        if self.q_norm_w is not None:
            for name, w, n in (("q", self.q_norm_w, H), ("k", self.k_norm_w, G)):
                n = n if self.qk_norm == "whole" else 1
                out[name + ".norm"] = ((n * D,), _pad_heads(w, n, D, self.dp))
        if self.rot_order is not None:
            for name, (shape, put) in list(out.items()):
                if name[0] in "qk":
                    out[name] = (shape, lambda t, put=put: put(self._reordered(t)))
        if self.key_bias is not None:
            out["pb"] = ((H,), self.key_bias.data.copy_)
        if self.head_gate:
            out["g"] = ((H, width), lambda t: load_in(t, self.g_off))
        return out

    # ---- forward -------------------------------------------------------------------------------------------
    def mix(self, p: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor, kept: dict) -> None:
        q = rt.buffer("query", p.shape[0], self.k_off)
        own = (kept["k"], kept["v"]) if self.kv_from is None else (None, None)
        hops.qkv_prep(p, self.heads, self.own_kv, self.dim, self.vdim, q, *own, meta, self.conv_w, kept.get("conv"), self.qk_norm, self.q_norm_w, self.k_norm_w, self.eps, self.temp_coef,
                      self.temp_every, self.cos_sin)
        hops.grouped_attention(q, kept["k"], kept["v"], out, meta, self.heads, self.kv_heads, self.scale, self.slopes,
                               self.sink, self.out_scale, rt.sm_count, window=self.window, keep=self.keep,
                               key_bias=self.key_bias, chunk=self.chunk, gate=p[:, self.g_off:] if self.head_gate else None)


class LightningAttention(Part):
    """Linear attention with a fixed decay per head: ``S <- decay S + k v^T``, ``o = S^T q`` on ``silu`` of the projected
    queries, keys and values (fp32 state), then one RMS norm over the concatenated heads with a weight, times
    ``sigmoid(W_g x)`` and ``out_scale``. It is the state-space recurrence with unit steps, one group per head and no
    skip, and runs on the same kernels."""
    recurrent = True

    def __init__(self, sizes: dict, eps: float, *, dtype, device, out_scale: float = 1.0):
        super().__init__()
        self.heads, self.dim, self.vdim = (int(sizes[k]) for k in ("heads", "dim", "vdim"))
        self.decays = [float(d) for d in sizes["decay"]]
        if len(self.decays) != self.heads or not all(0.0 <= d <= 1.0 for d in self.decays):
            raise ValueError(f"{self.heads} decays between 0 and 1 are needed, got {self.decays}")
        self.eps, self.dtype, self.device, self.out_scale = eps, dtype, torch.device(device), float(out_scale)
        self.dp, self.vp = pad8(self.dim), pad8(self.vdim)
        H = self.heads
        # [values | keys | queries | gate]: the first three in the order of the recurrence's kernels
        self.k_off, self.q_off, self.g_off = H * self.vp, H * (self.vp + self.dp), H * (self.vp + 2 * self.dp)
        self.in_cols, self.out_cols, self.silu_cols = self.g_off + H * self.vp, H * self.vp, self.g_off
        self.norm_w = _vec(H * self.vp, dtype, device, 0.0)
        self.decay: Optional[torch.Tensor] = None

    def bind_runtime(self, rt) -> None:
        self.decay = torch.tensor(self.decays, dtype=torch.float32, device=self.device)

    def workspaces(self) -> list[tuple[str, int]]:
        return [("recurrent", self.out_cols)]

    def state_bytes_per_slot(self) -> int:
        return 4 * self.heads * self.vp * self.dp

    def init_state(self, kept: dict, num_slots: int) -> None:
        kept["state"] = torch.zeros(num_slots, self.heads, self.vp, self.dp, dtype=torch.float32, device=self.device)

    def tensor_targets(self, width: int, load_in, load_bias, load_out) -> dict:
        H, D, V = self.heads, self.dim, self.vdim
        return {
            "q": ((H * D, width), _by_head(load_in, D, self.dp, self.q_off)),
            "k": ((H * D, width), _by_head(load_in, D, self.dp, self.k_off)),
            "v": ((H * V, width), _by_head(load_in, V, self.vp, 0)),
            "g": ((H * V, width), _by_head(load_in, V, self.vp, self.g_off)),
            "norm": ((H * V,), _pad_heads(self.norm_w, H, V, self.vp)),
            "o": ((width, H * V), lambda t: _by_head(lambda r, i: load_out(r.t(), i), V, self.vp, 0)(t.t())),
        }

    @property
    def chunkable(self) -> bool:
        return self.device.type == "cuda" and hops.ssd_chunkable(self.dtype, self.vp, self.dp)

    def mix(self, p: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor, kept: dict) -> None:
        y, e = rt.buffer("recurrent", p.shape[0], self.out_cols), meta.extra
        for run, seqs in ((hops.decay_scan, e["scan_seqs"]),
                          (hops.decay_chunk if self.chunkable else hops.decay_scan, e["chunk_seqs"])):
            run(p, self.decay, kept["state"], y, seqs, meta.cu_q, meta.kv_lens, e["state_slots"])
        hops.norm_gate(y, p[:, self.g_off:], self.norm_w, self.heads * self.vdim, self.eps, self.out_scale, out)


class GatedMLP(nn.Module):
    """The first half of a gated feed-forward, ``act(W_gate x) * (W_up x)``, as a part of a :class:`SumMixer` (whose output
    projection holds ``W_down``). ``act``: "silu" or "gelu_tanh"."""

    def __init__(self, sizes: dict, width: int, *, dtype, device):
        super().__init__()
        self.ff, self.width, self.act = int(sizes["ff"]), width, str(sizes["act"])
        self.out_cols = pad8(self.ff)
        self.gate_up = PaddedLinear(width, 2 * self.out_cols, dtype=dtype, device=device)

    def workspaces(self) -> list[tuple[str, int]]:
        # the fp32 product has no gated form: its two halves go through a buffer
        return [("gate_up", 2 * self.out_cols)] if self.gate_up.weight.dtype == torch.float32 else []

    def tensor_targets(self, load_out) -> dict:
        return {"gate": ((self.ff, self.width), lambda t: self.gate_up.load_rows(t, 0)),
                "up": ((self.ff, self.width), lambda t: self.gate_up.load_rows(t, self.out_cols)),
                "down": ((self.width, self.ff), lambda t: load_out(t, 0))}

    def forward(self, x: torch.Tensor, rt, out: torch.Tensor) -> None:
        w = self.gate_up.weight
        tmp = rt.buffer("gate_up", x.shape[0], w.shape[0]) if w.dtype == torch.float32 else None
        hops.gated_product(x, w, self.act, out, tmp)


PARTS = {"grouped_attention": GroupedAttention, "lightning_attention": LightningAttention}


class SumMixer(Mixer):
    """The sum of its parts (and of a gated feed-forward), all of the same input. ``sizes`` = {"parts": {name: {"kind",
    "sizes", "options"}}}; the checkpoint names of a part's tensors have ``<name>.`` in front, or nothing for the name
    "". One matrix product makes every part's projected input, one more the feed-forward's, and the last one takes the
    parts' results side by side, so that their sum is its accumulation."""

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device, mlp: Optional[dict] = None):
        super().__init__()
        self.width = width
        self.parts = nn.ModuleDict()
        for name, spec in sizes["parts"].items():
            self.parts[name or "only"] = PARTS[spec["kind"]](spec["sizes"], eps, dtype=dtype, device=device,
                                                             **spec.get("options", {}))
        self.prefix = {name or "only": name + "." if name else "" for name in sizes["parts"]}
        self.glu = GatedMLP(mlp, width, dtype=dtype, device=device) if mlp is not None else None
        self.in_at, self.out_at, i, o = {}, {}, 0, 0
        for name, part in self.parts.items():
            self.in_at[name], self.out_at[name] = (i, i + part.in_cols), (o, o + part.out_cols)
            i, o = i + part.in_cols, o + part.out_cols
        self.glu_at = (o, o + self.glu.out_cols) if self.glu is not None else (o, o)
        self.in_proj = PaddedLinear(width, i, bias=any(p.biased for p in self.parts.values()), dtype=dtype, device=device)
        self.out_proj = PaddedLinear(self.glu_at[1], width, dtype=dtype, device=device)
        silu = [(self.in_at[n][0], self.in_at[n][0] + p.silu_cols) for n, p in self.parts.items() if p.silu_cols]
        if len(silu) > 1:
            raise ValueError("one part per mixer may ask for silu on its projection")
        self.silu = silu[0] if silu else None
        self.recurrent = any(p.recurrent for p in self.parts.values())
        self.attends = any(p.attends for p in self.parts.values())

    @property
    def tileable(self) -> bool:
        return all(p.tileable for p in self.parts.values() if p.attends)

    def workspaces(self) -> list[tuple[str, int]]:
        out = [("proj", self.in_proj.out_padded), ("mixed", self.out_proj.in_padded)]
        for part in list(self.parts.values()) + ([self.glu] if self.glu is not None else []):
            out += part.workspaces()
        return out

    def cache_bytes_per_block(self, block_size: int) -> int:
        return sum(p.cache_bytes_per_block(block_size) for p in self.parts.values())

    def state_bytes_per_slot(self) -> int:
        return sum(p.state_bytes_per_slot() for p in self.parts.values())

    def new_kept(self) -> dict:
        return {name: {} for name in self.parts}

    def init_cache(self, kept: dict, num_blocks: int, block_size: int) -> None:
        for name, part in self.parts.items():
            part.init_cache(kept[name], num_blocks, block_size)

    def kv_sources(self) -> dict:
        """part -> the layer whose part of that name keeps its keys and values"""
        return {n: p.kv_from for n, p in self.parts.items() if getattr(p, "kv_from", None) is not None}

    def share_cache(self, name: str, kept: dict, source_kept: dict) -> None:
        kept[name].update((k, source_kept[name][k]) for k in ("k", "v"))

    def init_state(self, kept: dict, num_slots: int) -> None:
        for name, part in self.parts.items():
            part.init_state(kept[name], num_slots)

    def bind_runtime(self, rt) -> None:
        for part in self.parts.values():
            part.bind_runtime(rt)

    def launch_key(self, meta: AttentionMetadata, block_size: int, sm_count: int) -> tuple:
        return tuple(p.launch_key(meta, block_size, sm_count) for p in self.parts.values())

    def tensor_targets(self) -> dict:
        out = {}
        for name, part in self.parts.items():
            i, o = self.in_at[name][0], self.out_at[name][0]

            def load_bias(t, row, i=i):
                self.in_proj.bias.data[i + row:i + row + t.shape[0]].copy_(t)
            targets = part.tensor_targets(self.width, lambda t, row, i=i: self.in_proj.load_rows(t, i + row), load_bias,
                                          lambda t, col, o=o: self.out_proj.load_cols(t, o + col))
            out.update({self.prefix[name] + k: v for k, v in targets.items()})
        return out

    def mlp_targets(self) -> dict:
        """Tensors of the feed-forward (behind ``<layer>.mlp.``)."""
        return self.glu.tensor_targets(lambda t, col: self.out_proj.load_cols(t, self.glu_at[0] + col))

    def forward(self, x: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor, kept: dict) -> None:
        n = x.shape[0]
        mixed = rt.buffer("mixed", n, self.out_proj.in_padded)
        if self.glu is not None:
            self.glu(x, rt, mixed[:, self.glu_at[0]:self.glu_at[1]])
        p = hops.projection(x, self.in_proj.weight, self.in_proj.bias, self.silu,
                            rt.buffer("proj", n, self.in_proj.out_padded))
        for name, part in self.parts.items():
            (i0, i1), (o0, o1) = self.in_at[name], self.out_at[name]
            part.mix(p[:, i0:i1], meta, rt, mixed[:, o0:o1], kept[name])
        self.out_proj(mixed, out=out)


MIXERS = {"latent_attention": LatentAttention, "mamba2": Mamba2Mixer, "mingru": MinGRUMixer, "sum": SumMixer}
FEED_FORWARDS = {"dense": PolyNormMLP, "activated": ActMLP, "routed": RoutedMLP}

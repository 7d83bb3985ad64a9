"""Token mixers and feed-forwards of hybrid decoders: layers that a model's configuration lists one by one, each with
its own kind and sizes (``models/hybrid.py``).

A mixer owns its weights and whatever it keeps between steps - pages of a cache (``cache_bytes_per_block`` /
``init_cache``) or a slot of recurrent state per sequence (``state_bytes_per_slot`` / ``init_state``) - and maps
activation rows to sublayer outputs: ``forward(x, meta, rt, out)``. All sizes and constants are parameters, so
another design can list the same mixers with other values. :data:`MIXERS` and :data:`FEED_FORWARDS` are the names a
configuration may use.

Activations and weights are bf16 or fp32 (the engine's dtype); norms, rotary angles, attention scores and softmax,
decays and recurrent state are fp32 in both.
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn

from ..ops import hybrid as hops
from ..ops import reference
from .attention import AttentionMetadata
from .linear import PaddedLinear, pad8


def _vec(n: int, dtype, device, fill: float = 1.0) -> nn.Parameter:
    return nn.Parameter(torch.full((n,), fill, dtype=dtype, device=device), requires_grad=False)


class Mixer(nn.Module):
    recurrent = False            # keeps a state slot per sequence

    def cache_bytes_per_block(self, block_size: int) -> int:
        return 0

    def state_bytes_per_slot(self) -> int:
        return 0

    def init_cache(self, num_blocks: int, block_size: int) -> None:
        pass

    def init_state(self, num_slots: int) -> None:
        pass

    def state_tensors(self) -> list[torch.Tensor]:
        """Every tensor kept between steps."""
        return []

    def drop_state(self) -> None:
        pass

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
    """

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device, max_positions: int, gated: bool = True):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim = (int(sizes[k]) for k in ("heads", "dim", "rot_dim", "vdim"))
        self.kv_rank, self.q_rank = int(sizes["kv_rank"]), int(sizes["q_rank"])
        self.scale, self.eps, self.width, self.gated = float(sizes["scale"]), eps, width, gated
        self.rot = dict(sizes["rot"])
        self.rot_dims = int(self.rot["dims"])
        if self.rot_dims % 2 or not 0 < self.rot_dims <= self.rot_dim:
            raise ValueError(f"rotated dimensions {self.rot_dims} do not fit a part of {self.rot_dim}")
        self.max_positions = max_positions
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
        self.cache: Optional[torch.Tensor] = None
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
                                       self.o_proj.weight.dtype, meta.max_kv_len, sm_count)

    # ---- cache -----------------------------------------------------------------------------------------
    def cache_bytes_per_block(self, block_size: int) -> int:
        return block_size * self.row * self.o_proj.weight.element_size()

    def init_cache(self, num_blocks: int, block_size: int) -> None:
        w = self.o_proj.weight
        self.cache = torch.zeros(num_blocks, block_size, self.row, dtype=w.dtype, device=w.device)

    def state_tensors(self) -> list[torch.Tensor]:
        return [] if self.cache is None else [self.cache]

    def drop_state(self) -> None:
        self.cache = None

    def rope_key(self) -> tuple:
        s = self.rot.get("scaling")
        return (self.rot_dims, float(self.rot["base"]), tuple(sorted((s or {}).items())))

    def make_rope_table(self) -> torch.Tensor:
        import math
        s = self.rot.get("scaling")
        scaling = None
        if s:
            factor = float(s["factor"])
            scaling = dict(rope_type="yarn", factor=factor, original_max_position_embeddings=float(s["original"]),
                           beta_fast=float(s["fast"]), beta_slow=float(s["slow"]),
                           attention_factor=0.1 * math.log(factor) + 1.0)
        return reference.build_cos_sin_cache(self.rot_dims, self.max_positions, float(self.rot["base"]), scaling,
                                             self.o_proj.weight.device)

    # ---- weights ---------------------------------------------------------------------------------------
    def tensor_targets(self) -> dict:
        H, D, V, R, Q, W = self.heads, self.dim, self.vdim, self.kv_rank, self.q_rank, self.width

        def uk(t):
            self.ukv_proj.load_rows(t, 0)
            self.ukt_w.data[:, :, :D].copy_(t.view(H, D, R).transpose(1, 2))
        out = {
            "dq": ((Q, W), lambda t: self.in_proj.load_rows(t, 0)),
            "dq.norm": ((Q,), self.q_norm_w.data.copy_),
            "uq": ((H * (D + self.rot_dim), Q), lambda t: self.uq_proj.load_rows(t, 0)),
            "dkv": ((R + self.rot_dim, W), lambda t: self.in_proj.load_rows(t, self.kv_off)),
            "dkv.norm": ((R,), self.kv_norm_w.data.copy_),
            "uk": ((H * D, R), uk),
            "uv": ((H * V, R), lambda t: self.ukv_proj.load_rows(t, H * D)),
            "o": ((W, H * V), lambda t: self.o_proj.load_rows(t, 0)),
        }
        if self.gated:
            out["g"] = ((H * V, W), lambda t: self.in_proj.load_rows(t, self.gate_off))
        return out

    # ---- forward ---------------------------------------------------------------------------------------
    def forward(self, x: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor) -> None:
        n, H = x.shape[0], self.heads
        p = self.in_proj(x, out=rt.buffer("proj", n, self.in_proj.out_padded))
        cq = rt.buffer("latent_q", n, self.uq_proj.in_padded)
        hops.latent_prep(p, 0, self.q_rank, self.q_norm_w, cq, self.kv_off, self.kv_rank, self.kv_norm_w, self.rot_dim,
                         self.rot_dims, self.cos_sin, meta.positions, meta.slot_mapping, self.cache, self.eps)
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
            hops.latent_attention(qa, self.cache, meta.tok_seq, meta.tok_kvlen, m, meta.block_table, self.kv_rank,
                                  self.scale, o, meta.max_kv_len, rt.sm_count)
            hops.latent_values(o, meta.tok_row, w_uv, H, self.vdim, self.kv_rank, gate, attn)
        if meta.num_tiles:
            # keys and values of the tiles' contexts (the step's own tokens are in the cache already)
            rows = meta.extra_cpu["ctx_rows"]
            lat = rt.buffer("ctx_latent", rows, self.row)
            hops.latent_gather(self.cache, meta.extra["ctx_seqs"], meta.extra["ctx_cu"], meta.extra_cpu["ctx_max"],
                               meta.block_table, lat)
            kv = self.ukv_proj(lat[:, :self.ukv_proj.in_padded], out=rt.buffer("ctx_kv", rows, self.ukv_proj.out_padded))
            hops.rope_tail_(q, H, self.dim + self.rot_dim, self.dim, self.rot_dims, self.cos_sin, meta.positions)
            hops.latent_prefill(q, kv, lat, pad8(self.kv_rank), rows, meta.extra["ctx_begin"], attn, gate, meta.cu_q,
                                meta.kv_lens, meta.tile_seq, meta.tile_q0, meta.num_tiles, H, self.dim, self.rot_dim,
                                self.vdim, self.scale)
        self.o_proj(attn, out=out)


class Mamba2Mixer(Mixer):
    """Mamba-2: projection to [gate z | x, B, C | step sizes], causal convolution + silu of x, B and C, state-space
    recurrence per head with an fp32 state, skip ``D x``, gate, grouped RMS norm, output projection."""
    recurrent = True

    def __init__(self, sizes: dict, width: int, eps: float, *, dtype, device, max_positions: int = 0):
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
        self.state: Optional[torch.Tensor] = None        # [slots, heads, vdim, N] fp32
        self.conv_state: Optional[torch.Tensor] = None   # [slots, taps - 1, channels]

    def workspaces(self) -> list[tuple[str, int]]:
        return [("proj", self.in_proj.out_padded), ("conv", pad8(self.channels)), ("mixed", self.o_proj.in_padded),
                ("gated", self.o_proj.in_padded)]

    @property
    def chunkable(self) -> bool:
        return self.conv_w.is_cuda and hops.ssd_chunkable(self.conv_w.dtype, self.vdim, self.N)

    # ---- state -----------------------------------------------------------------------------------------
    def state_bytes_per_slot(self) -> int:
        return 4 * self.inner * self.N + (self.taps - 1) * self.channels * self.conv_w.element_size()

    def init_state(self, num_slots: int) -> None:
        dev = self.conv_w.device
        self.state = torch.zeros(num_slots, self.heads, self.vdim, self.N, dtype=torch.float32, device=dev)
        self.conv_state = torch.zeros(num_slots, self.taps - 1, self.channels, dtype=self.conv_w.dtype, device=dev)

    def state_tensors(self) -> list[torch.Tensor]:
        return [] if self.state is None else [self.state, self.conv_state]

    def drop_state(self) -> None:
        self.state = self.conv_state = None

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
    def forward(self, x: torch.Tensor, meta: AttentionMetadata, rt, out: torch.Tensor) -> None:
        n = x.shape[0]
        p = self.in_proj(x, out=rt.buffer("proj", n, self.in_proj.out_padded))
        xbc = rt.buffer("conv", n, pad8(self.channels))
        e = meta.extra
        hops.causal_conv(p[:, self.x_off:], self.conv_w, self.conv_b, self.conv_state, xbc, e["row_seq"], meta.cu_q,
                         meta.kv_lens, e["state_slots"], meta.all_single)
        y = rt.buffer("mixed", n, self.o_proj.in_padded)
        # long runs in chunks on the tensor cores (sizes permitting), everything else token by token
        for run, seqs in ((hops.ssd_scan, e["scan_seqs"]),
                          (hops.ssd_chunk if self.chunkable else hops.ssd_scan, e["chunk_seqs"])):
            run(xbc, p[:, self.dt_off:], self.dt_bias, self.A_log, self.D, self.state, y, seqs, meta.cu_q, meta.kv_lens,
                e["state_slots"], self.groups)
        g = rt.buffer("gated", n, self.o_proj.in_padded)
        hops.gated_group_norm(y, p, self.norm_w, self.norm_groups, self.eps, g)
        self.o_proj(g, out=out)


class PolyNormMLP(nn.Module):
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


MIXERS = {"latent_attention": LatentAttention, "mamba2": Mamba2Mixer}
FEED_FORWARDS = {"dense": PolyNormMLP}

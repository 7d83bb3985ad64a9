"""Decoder whose layers are listed one by one in the configuration, each with a mixer (attention with pages of a cache,
or a recurrence with a state slot per sequence) and an optional feed-forward (``layers/mixers.py``).

Differences from :class:`~tokenweave_b200.models.decoder.DecoderModel`, whose interface towards the worker and the model
runner this class shares:

* the residual stream is fp32 and the sublayers read it directly (in the activation type); the RMS norm is applied to
  a sublayer's OUTPUT before the sum: ``x += norm(f(x))``. Sum, norm, and the cast of the next input (or the model's
  final norm) are one kernel;
* bf16 and fp32 both run on the GPU (the fp32 mode in true fp32);
* one GPU: a norm on the sublayer's output needs the whole output, so the fused reduce-scatter + add + norm of the
  pre-norm families does not apply, and tensor / pipeline parallelism are refused.
"""
from __future__ import annotations

from typing import Iterable, Optional

import numpy as np
import torch
from torch import nn

from ..config import ModelConfig
from ..layers.attention import PREFILL_MIN_Q, AttentionMetadata
from ..layers.linear import PaddedLinear, pad8
from ..layers.mixers import FEED_FORWARDS, MIXERS, LatentAttention
from ..ops import hybrid as hops
from ..parallel.comm import TPCommunicator
from ..parallel.state import get_tp
from ..parallel.symm_mem import create_symmetric_buffer


class HybridRuntime:
    """Buffers shared by all layers: the fp32 residual stream, the activation rows, and named workspaces that grow to
    the widest layer's need and are carved from one allocation each (zeroed once: pad columns stay zero because every
    user of a workspace with the same width writes the same columns)."""

    def __init__(self, cfg: ModelConfig, max_tokens: int, device: torch.device, tw_cfg, provider: Optional[str] = None):
        tp = get_tp()
        self.device, self.max_tokens = device, max_tokens
        w8 = pad8(cfg.hidden_size)
        self.staging = create_symmetric_buffer(max_tokens, w8, cfg.dtype, tp, provider,
                                               tw_cfg.transport in ("auto", "multimem"))
        self.hidden = self.staging.tensor
        self.hidden.zero_()
        self.residual = torch.zeros(max_tokens, w8, dtype=torch.float32, device=device)
        self.sublayer = torch.zeros(max_tokens, w8, dtype=cfg.dtype, device=device)
        self.comm = TPCommunicator(self.staging, tp, tw_cfg.wait_budget_ms, tw_cfg.transport)
        self.dtype = cfg.dtype
        self.sm_count = torch.cuda.get_device_properties(device).multi_processor_count if device.type == "cuda" else 0
        # context tokens whose keys and values a step may expand
        self.context_rows = max(max_tokens, min(cfg.max_model_len, 32768))
        self.rope_tables: dict = {}
        self._buffers: dict[tuple, torch.Tensor] = {}

    def buffer(self, name: str, rows: int, cols: int) -> torch.Tensor:
        """``[rows, cols]`` workspace in the activation type. Buffers are made once per (name, width) for the step's
        token budget and never freed, so their addresses are stable for captured graphs."""
        key = (name, cols)
        t = self._buffers.get(key)
        if t is None or t.shape[0] < rows:
            t = self._buffers[key] = torch.zeros(max(rows, self.max_tokens), cols, dtype=self.dtype, device=self.device)
        return t[:rows]


class HybridLayer(nn.Module):
    def __init__(self, spec: dict, cfg: ModelConfig, *, device):
        super().__init__()
        kind = spec["type"]
        if kind not in MIXERS:
            raise ValueError(f"unknown mixer {kind!r} (known: {sorted(MIXERS)})")
        W, eps, dt = cfg.hidden_size, cfg.rms_norm_eps, cfg.dtype
        self.mixer = MIXERS[kind](spec["mixer"], W, eps, dtype=dt, device=device, max_positions=cfg.max_model_len)
        self.norm1_w = nn.Parameter(torch.ones(W, dtype=dt, device=device), requires_grad=False)
        self.mlp = self.norm2_w = None
        mlp = spec.get("mlp")
        if mlp is not None:
            if mlp["kind"] not in FEED_FORWARDS:
                raise ValueError(f"unknown feed-forward {mlp['kind']!r} (known: {sorted(FEED_FORWARDS)})")
            self.mlp = FEED_FORWARDS[mlp["kind"]](mlp, W, eps, dtype=dt, device=device)
            self.norm2_w = nn.Parameter(torch.ones(W, dtype=dt, device=device), requires_grad=False)

    def tensor_targets(self) -> dict:
        W = self.norm1_w.numel()
        out = {"norm1": ((W,), self.norm1_w.data.copy_)}
        out.update({f"mix.{k}": v for k, v in self.mixer.tensor_targets().items()})
        if self.mlp is not None:
            out["norm2"] = ((W,), self.norm2_w.data.copy_)
            out.update({f"mlp.{k}": v for k, v in self.mlp.tensor_targets().items()})
        return out


class HybridDecoder(nn.Module):
    architecture = "hybrid"

    def __init__(self, cfg: ModelConfig, *, device, embedding_parallel: bool = False):
        super().__init__()
        tp = get_tp()
        if tp.world_size > 1 or tp.pp_size > 1:
            raise ValueError(f"{cfg.architecture} runs on one GPU: no tensor or pipeline parallelism")
        if not cfg.layers:
            raise ValueError("a hybrid decoder needs the list of its layers")
        self.cfg = cfg
        dt, W = cfg.dtype, cfg.hidden_size
        self.embed_w = nn.Parameter(torch.zeros(cfg.vocab_size, pad8(W), dtype=dt, device=device), requires_grad=False)
        self.layers = nn.ModuleList([HybridLayer(s, cfg, device=device) for s in cfg.layers])
        self.final_norm_w = nn.Parameter(torch.ones(W, dtype=dt, device=device), requires_grad=False)
        self.head = PaddedLinear(W, cfg.vocab_size, dtype=dt, device=device)
        self.rt: Optional[HybridRuntime] = None
        latent = [l.mixer for l in self.layers if isinstance(l.mixer, LatentAttention)]
        self.expand = bool(latent) and all(m.expandable for m in latent)      # long runs may use the expanded form
        self.recurrent = any(l.mixer.recurrent for l in self.layers)

    # ---- runtime ---------------------------------------------------------------------------------------
    def setup_runtime(self, max_tokens: int, tw_cfg, provider: Optional[str] = None,
                      disable_custom_all_reduce: bool = True) -> HybridRuntime:
        self.rt = HybridRuntime(self.cfg, max_tokens, self.final_norm_w.device, tw_cfg, provider)
        for layer in self.layers:
            m = layer.mixer
            for part in (m, layer.mlp):
                for name, cols in part.workspaces() if part is not None else ():
                    self.rt.buffer(name, max_tokens, cols)
                if self.expand and part is m and isinstance(m, LatentAttention):
                    for name, cols in m.context_workspaces():
                        self.rt.buffer(name, self.rt.context_rows, cols)
            if isinstance(m, LatentAttention):
                key = m.rope_key()
                if key not in self.rt.rope_tables:
                    self.rt.rope_tables[key] = m.make_rope_table()
                m.cos_sin = self.rt.rope_tables[key]
        return self.rt

    def kv_cache_bytes_per_block(self, block_size: int) -> int:
        return max(1, sum(l.mixer.cache_bytes_per_block(block_size) for l in self.layers))

    def state_bytes_per_slot(self) -> int:
        return sum(l.mixer.state_bytes_per_slot() for l in self.layers)

    def init_kv_cache(self, num_blocks: int, block_size: int) -> None:
        for l in self.layers:
            l.mixer.init_cache(num_blocks, block_size)

    def init_state(self, num_slots: int) -> None:
        for l in self.layers:
            l.mixer.init_state(num_slots)

    def cache_tensors(self) -> list[torch.Tensor]:
        return [t for l in self.layers for t in l.mixer.state_tensors()]

    def drop_caches(self) -> None:
        for l in self.layers:
            l.mixer.drop_state()

    # ---- a step's layout -------------------------------------------------------------------------------
    def plan_step(self, q_lens, kv_lens, state_slots):
        """Routing of a step's rows: (attention plan as of ``plan_attention``, extra int32 arrays, host values).

        Attention: a run of a prompt goes to 128-query tiles over expanded keys and values when it is long enough to
        pay for expanding its context (a product over the whole context, whatever the run's length), and when the
        context fits the workspace; every other row is attended alone in the absorbed form. Recurrences: long runs in
        chunks, short ones token by token."""
        B = len(q_lens)
        if max(q_lens) == 1:
            rows = np.arange(B, dtype=np.int32)
            plan = ([], [], rows, rows, np.asarray(kv_lens, dtype=np.int32))
            extra = {"row_seq": rows}
            if self.recurrent:
                extra.update(state_slots=np.asarray(state_slots, dtype=np.int32), scan_seqs=rows, chunk_seqs=rows[:0])
            return plan, extra, {}
        n = np.asarray(q_lens)
        tiled, ctx_rows = [], 0
        if self.expand:
            for b, (ql, kv) in enumerate(zip(q_lens, kv_lens)):
                if (ql >= 64 or (ql >= PREFILL_MIN_Q and kv <= 2 * ql)) and ctx_rows + kv <= self.rt.context_rows:
                    tiled.append(b)
                    ctx_rows += kv
        row_seq = np.repeat(np.arange(B, dtype=np.int32), n)
        start = np.cumsum(n) - n
        tok_row = np.flatnonzero(~np.isin(row_seq, tiled)).astype(np.int32)
        tok_seq = row_seq[tok_row]
        tok_kv = (np.asarray(kv_lens) - n)[tok_seq] + (tok_row - start[tok_seq]) + 1
        tile_seq = [b for b in tiled for _ in range(0, q_lens[b], 128)]
        tile_q0 = [q0 for b in tiled for q0 in range(0, q_lens[b], 128)]
        order = np.argsort([-(kv_lens[b] - q_lens[b] + q0) for b, q0 in zip(tile_seq, tile_q0)], kind="stable")
        plan = ([tile_seq[i] for i in order], [tile_q0[i] for i in order], tok_row, tok_seq, tok_kv.astype(np.int32))
        extra, host = {"row_seq": row_seq}, {}
        if tiled:
            cu = np.zeros(len(tiled) + 1, dtype=np.int32)
            np.cumsum([kv_lens[b] for b in tiled], out=cu[1:])
            begin = np.full(B, -1, dtype=np.int32)
            begin[tiled] = cu[:-1]
            extra.update(ctx_seqs=np.asarray(tiled, dtype=np.int32), ctx_cu=cu, ctx_begin=begin)
            host = {"ctx_rows": int(cu[-1]), "ctx_max": max(kv_lens[b] for b in tiled)}
        if self.recurrent:
            long = n >= hops.CHUNK_MIN_TOKENS
            extra.update(state_slots=np.asarray(state_slots, dtype=np.int32),
                         scan_seqs=np.flatnonzero(~long).astype(np.int32), chunk_seqs=np.flatnonzero(long).astype(np.int32))
        return plan, extra, host

    def launch_key(self, meta: AttentionMetadata, block_size: int) -> tuple:
        """What shapes a step's launches besides its token and sequence counts (part of a graph's signature)."""
        return (meta.all_single, tuple(sorted(meta.extra_cpu.items())),
                tuple(sorted((k, v.shape[0]) for k, v in meta.extra.items())),
                tuple(sorted({l.mixer.launch_key(meta, block_size, self.rt.sm_count) for l in self.layers
                              if isinstance(l.mixer, LatentAttention)})))

    # ---- forward ---------------------------------------------------------------------------------------
    @torch.inference_mode()
    def forward(self, step) -> torch.Tensor:
        """Runs the stack; returns the final-norm rows ``[T, padded width]``."""
        rt, cfg, meta = self.rt, self.cfg, step.meta
        T, eps = step.plan.num_tokens, cfg.rms_norm_eps
        x32, xa, y = rt.residual[:T], rt.hidden[:T], rt.sublayer[:T]
        hops.embed_residual(step.input_ids, self.embed_w, x32, xa, cfg.hidden_size)
        last = self.layers[-1]
        for layer in self.layers:
            layer.mixer(xa, meta, rt, y)
            final = self.final_norm_w if layer is last and layer.mlp is None else None
            hops.postnorm_add_(y, x32, layer.norm1_w, eps, xa, final)
            if layer.mlp is not None:
                layer.mlp(xa, rt, y)
                hops.postnorm_add_(y, x32, layer.norm2_w, eps, xa, self.final_norm_w if layer is last else None)
        return xa

    @torch.inference_mode()
    def compute_logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """fp32 logits ``[rows, vocab]``."""
        return self.head(hidden_rows)[:, : self.cfg.vocab_size].float() * self.cfg.logit_scale

    # ---- weights ---------------------------------------------------------------------------------------
    def tensor_targets(self) -> dict:
        V, W = self.cfg.vocab_size, self.cfg.hidden_size
        out = {"embed": ((V, W), lambda t: self.embed_w.data[:, :W].copy_(t)),
               "final.norm": ((W,), self.final_norm_w.data.copy_),
               "head": ((V, W), lambda t: self.head.load_rows(t, 0))}
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.tensor_targets().items()})
        return out

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        """Tensors by their names in the checkpoint (``embed``, ``l<i>.mix.<name>``, ``l<i>.mlp.<name>``,
        ``l<i>.norm1`` ...). Every tensor of the design must come, in its shape; layers beyond the configured ones
        (a reduced layer count) are skipped."""
        targets = self.tensor_targets()
        loaded: set[str] = set()
        for name, t in weights:
            if name not in targets:
                head = name.split(".", 1)[0]
                if head[:1] == "l" and head[1:].isdigit() and int(head[1:]) >= len(self.layers):
                    continue
                raise ValueError(f"unexpected tensor {name!r} in a {self.cfg.architecture} checkpoint")
            shape, put = targets[name]
            if tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {tuple(shape)}")
            put(t)
            loaded.add(name)
        missing = sorted(set(targets) - loaded)
        if missing:
            raise ValueError(f"the checkpoint lacks {len(missing)} tensors (first: {missing[0]})")
        return loaded

    def init_dummy_weights(self, seed: int = 0) -> None:
        """Random weights of a plausible scale (performance runs): matrices N(0, init_std), unit norms, decays and
        step sizes in the usual state-space ranges."""
        g = torch.Generator(device=self.final_norm_w.device)
        g.manual_seed(seed)
        dev = self.final_norm_w.device

        def fill(name, shape):
            t = torch.empty(shape, dtype=torch.float32, device=dev)
            leaf = name.split(".mix.")[-1]
            if name.endswith(("norm", "norm1", "norm2")) or leaf == "D":
                return t.fill_(1.0)
            if leaf == "A_log":
                return t.uniform_(1.0, 16.0, generator=g).log_()
            if leaf == "dt_bias":
                return t.uniform_(-6.9, -2.3, generator=g)
            if leaf == "conv.b":
                return t.zero_()
            if leaf == "conv":
                return t.normal_(0.0, shape[1] ** -0.5, generator=g)
            if name.endswith(".mlp.act"):
                return torch.tensor([1 / 3, 1 / 3, 1 / 3, 0.0], device=dev)
            return t.normal_(0.0, self.cfg.init_std, generator=g)
        for name, (shape, put) in self.tensor_targets().items():
            put(fill(name, shape))

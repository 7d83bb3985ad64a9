"""Decoder whose layers are listed one by one in the configuration, each with a mixer (attention with pages of a cache,
or a recurrence with a state slot per sequence) and an optional feed-forward (``layers/mixers.py``).

Differences from :class:`~tokenweave_b200.models.decoder.DecoderModel`, whose interface towards the worker and the model
runner this class shares:

* the residual stream is fp32. ``ModelConfig.block`` says how a layer adds to it:
  "output_norm": the sublayers read the stream directly (in the activation type) and the RMS norm is applied to a
  sublayer's OUTPUT, ``x += norm1(mixer(x))``, ``x += norm2(ff(x))``; sum, norm, and the cast of the next input (or the
  model's final norm) are one kernel;
  "parallel": both sublayers read one norm of the stream, ``x += mixer(norm1(x)) + ff(norm1(x))``; the two results come
  out of one matrix product, and their addition and the next layer's norm (or the final one) are one kernel;
  "streams": hyper-connections - several residual streams, every sublayer reads the norm of a weighted sum of them and all
  streams are rebuilt from the old ones and the sublayer's output; that and the next sublayer's norm are one kernel (one
  stream with weights of one is the usual pre-norm block);
  "sandwich": a norm in front of every sublayer and one behind it, ``x += post(f(pre(x)))``; with ``depth_average`` a layer
  passes on a weighted sum of the embedding output and all layers' results so far, which are kept for the step; norm, sum,
  average and the next sublayer's norm are one kernel;
* a layer may read the keys and values that an earlier one keeps (``GroupedAttention``'s ``kv_from``);
* layers may be run several times in a row with the same weights (``ModelConfig.loop``); every pass keeps its own cache
  and state, and before each pass but the first the embedding output is added to the stream;
* a table of embeddings of token pairs may be added to the token embeddings (``ModelConfig.bigram``);
* bf16 and fp32 both run on the GPU (the fp32 mode in true fp32);
* one GPU: tensor / pipeline parallelism are refused (the fused reduce-scatter + add + norm of the pre-norm families
  works on a bf16 residual stream and neither on a norm of the sublayer's output nor on a sum with a stored row).
"""
from __future__ import annotations

from typing import Iterable, Optional

import numpy as np
import torch
from torch import nn

from ..config import ModelConfig
from ..layers.attention import PREFILL_MIN_Q, AttentionMetadata
from ..layers.linear import PaddedLinear, pad8
from ..layers.mixers import FEED_FORWARDS, MIXERS, LatentAttention, SumMixer
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
        self.residual = torch.zeros(max_tokens, max(1, cfg.streams) * w8, dtype=torch.float32, device=device)
        self.sublayer = torch.zeros(max_tokens, w8, dtype=cfg.dtype, device=device)
        # the embedding output and the results of the layers but the last, for averages over the depth
        self.results = (torch.zeros(cfg.num_layers, max_tokens, w8, dtype=torch.float32, device=device)
                        if cfg.depth_average else None)
        # the embedding output, for layers that run again
        self.first = torch.zeros(max_tokens, w8, dtype=torch.float32, device=device) if cfg.loop else None
        self.comm = TPCommunicator(self.staging, tp, tw_cfg.wait_budget_ms, tw_cfg.transport)
        self.dtype = cfg.dtype
        self.sm_count = torch.cuda.get_device_properties(device).multi_processor_count if device.type == "cuda" else 0
        # context tokens whose keys and values a step may expand
        self.context_rows = max(max_tokens, min(cfg.max_model_len, 32768))
        self.max_positions = cfg.max_model_len
        self.rope_tables: dict = {}
        self.tables: dict = {}              # bookkeeping that layers share, by the layers' own keys
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
    """``x += norm1(mixer(x))``, ``x += norm2(ff(x))``"""

    def __init__(self, spec: dict, cfg: ModelConfig, *, device):
        super().__init__()
        kind = spec["type"]
        if kind not in MIXERS:
            raise ValueError(f"unknown mixer {kind!r} (known: {sorted(MIXERS)})")
        W, eps, dt = cfg.hidden_size, cfg.rms_norm_eps, cfg.dtype
        self.mixer = MIXERS[kind](spec["mixer"], W, eps, dtype=dt, device=device, **spec.get("options", {}))
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


class ParallelLayer(nn.Module):
    """``x += mixer(norm1(x)) + ff(norm1(x))``: the mixer is a :class:`SumMixer` with the feed-forward as one more summand."""

    def __init__(self, spec: dict, cfg: ModelConfig, *, device):
        super().__init__()
        if spec["type"] != "sum":
            raise ValueError(f"a parallel block takes a sum of parts, not {spec['type']!r}")
        mlp = spec.get("mlp")
        if mlp is not None and mlp["kind"] != "gated":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r} in a parallel block")
        dt = cfg.dtype
        self.mixer = SumMixer(spec["mixer"], cfg.hidden_size, cfg.rms_norm_eps, dtype=dt, device=device, mlp=mlp)
        self.norm1_w = nn.Parameter(torch.ones(cfg.hidden_size, dtype=dt, device=device), requires_grad=False)
        self.mlp = None                     # part of the mixer

    def tensor_targets(self) -> dict:
        out = {"norm1": ((self.norm1_w.numel(),), self.norm1_w.data.copy_)}
        out.update({f"mix.{k}": v for k, v in self.mixer.tensor_targets().items()})
        if self.mixer.glu is not None:
            out.update({f"mlp.{k}": v for k, v in self.mixer.mlp_targets().items()})
        return out


class StreamLayer(HybridLayer):
    """Both sublayers of a layer read a norm of a weighted sum of the streams (``hops.streams_step``); ``hc[q]`` are the
    coefficients around sublayer q."""

    def __init__(self, spec: dict, cfg: ModelConfig, *, device):
        super().__init__(spec, cfg, device=device)
        S = max(1, cfg.streams)
        self.learned = cfg.streams > 0
        init = {"in": torch.ones(S), "out": torch.ones(S), "mix": torch.eye(S)}
        self.hc = nn.ModuleList(
            nn.ParameterDict({k: nn.Parameter(v.to(device=device, dtype=torch.float32, copy=True), requires_grad=False)
                              for k, v in init.items()}) for _ in range(1 if self.mlp is None else 2))

    def tensor_targets(self) -> dict:
        out = super().tensor_targets()
        if self.learned:
            for q, hc in enumerate(self.hc):
                out.update({f"hc{q + 1}.{k}": (tuple(v.shape), v.data.copy_) for k, v in hc.items()})
        return out


class Norm(nn.Module):
    """Weights of a layer norm ("layer": weight and bias) or an RMS norm ("rms": weight alone)."""

    def __init__(self, kind: str, width: int, dtype, device):
        super().__init__()
        if kind not in ("rms", "layer"):
            raise ValueError(f"unknown norm {kind!r}")
        vec = lambda fill: nn.Parameter(torch.full((width,), fill, dtype=dtype, device=device), requires_grad=False)
        self.w, self.b = vec(1.0), vec(0.0) if kind == "layer" else None

    @property
    def pair(self) -> tuple:
        return self.w, self.b

    def tensor_targets(self, name: str) -> dict:
        out = {name: ((self.w.numel(),), self.w.data.copy_)}
        if self.b is not None:
            out[name + ".b"] = ((self.b.numel(),), self.b.data.copy_)
        return out


class SandwichLayer(HybridLayer):
    """``x += norm1b(mixer(norm1(x)))``, ``x += norm2b(ff(norm2(x)))``; ``dwa[j]``: weight of result j (0: the embedding
    output, the last one: this layer's own) in what the layer passes on."""

    def __init__(self, spec: dict, cfg: ModelConfig, *, device, index: int):
        super().__init__(spec, cfg, device=device)
        self.norm1_w = self.norm2_w = None          # in ``norms``
        names = ("norm1", "norm1b") + (() if self.mlp is None else ("norm2", "norm2b"))
        self.norms = nn.ModuleDict({n: Norm(cfg.norm, cfg.hidden_size, cfg.dtype, device) for n in names})
        self.dwa = None
        if cfg.depth_average:
            own = torch.zeros(index + 2, dtype=torch.float32, device=device)
            own[-1] = 1.0
            self.dwa = nn.Parameter(own, requires_grad=False)

    def tensor_targets(self) -> dict:
        out = {f"mix.{k}": v for k, v in self.mixer.tensor_targets().items()}
        if self.mlp is not None:
            out.update({f"mlp.{k}": v for k, v in self.mlp.tensor_targets().items()})
        for name, norm in self.norms.items():
            out.update(norm.tensor_targets(name))
        if self.dwa is not None:
            out["dwa"] = (tuple(self.dwa.shape), self.dwa.data.copy_)
        return out


BLOCKS = {"output_norm": HybridLayer, "parallel": ParallelLayer, "streams": StreamLayer, "sandwich": SandwichLayer}


def layer_runs(num_layers: int, loop: Optional[dict]) -> list[tuple[int, bool]]:
    """(layer, a pass other than the first begins here) in the order in which the layers run."""
    if not loop:
        return [(i, False) for i in range(num_layers)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start < stop <= num_layers or times < 1:
        raise ValueError(f"a loop over layers {start} .. {stop - 1} of {num_layers}, {times} times")
    runs = [(i, False) for i in range(start)]
    for n in range(times):
        runs += [(i, n > 0 and i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, num_layers)]


def _tensors(kept: dict) -> list[torch.Tensor]:
    out = []
    for v in kept.values():
        out += _tensors(v) if isinstance(v, dict) else [v]
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
        self.head = PaddedLinear(W, cfg.vocab_size, dtype=dt, device=device)
        table = (self.head.weight.data[:cfg.vocab_size] if cfg.tie_word_embeddings
                 else torch.zeros(cfg.vocab_size, pad8(W), dtype=dt, device=device))
        self.embed_w = nn.Parameter(table, requires_grad=False)
        self.bigram_w = None
        if cfg.bigram:                      # one row per bucket, and one for tokens without a token before them
            self.bigram_w = nn.Parameter(torch.zeros(int(cfg.bigram["buckets"]) + 1, pad8(W), dtype=dt, device=device),
                                         requires_grad=False)
        sandwich = cfg.block == "sandwich"
        if not sandwich and (cfg.norm != "rms" or cfg.depth_average or cfg.embed_scale != 1.0):
            raise ValueError("layer norms, depth averages and an embedding scale are built for sandwich blocks")
        self.layers = nn.ModuleList([BLOCKS[cfg.block](s, cfg, device=device, **({"index": i} if sandwich else {}))
                                     for i, s in enumerate(cfg.layers)])
        self.runs = layer_runs(len(self.layers), cfg.loop)
        if cfg.block != "parallel" and (cfg.loop or cfg.bigram):
            raise ValueError("loops and pair embeddings are built for parallel blocks")
        self.kept = [self.layers[i].mixer.new_kept() for i, _ in self.runs]
        self.final_norm_w = nn.Parameter(torch.ones(W, dtype=dt, device=device), requires_grad=False)
        self.final_norm_b = (nn.Parameter(torch.zeros(W, dtype=dt, device=device), requires_grad=False)
                             if cfg.norm == "layer" else None)
        self._check_kv_sources()
        self.rt: Optional[HybridRuntime] = None
        mixers = [l.mixer for l in self.layers]
        latent = [m for m in mixers if isinstance(m, LatentAttention)]
        grouped = [m for m in mixers if isinstance(m, SumMixer) and m.attends]
        # long runs may go to query tiles: every attention of the model can take them; with latent attention their
        # contexts are expanded into a workspace first
        self.expand = bool(latent)
        # the keys an expanded run's first token sees: all of them, or the widest window's
        self.expand_window = 0 if any(not m.window for m in latent) else max((m.window for m in latent), default=0)
        self.tiles = (bool(latent or grouped) and all(m.expandable for m in latent) and all(m.tileable for m in grouped))
        self.recurrent = any(m.recurrent for m in mixers)

    def _kv_sources(self):
        """(layer, part, the layer whose keys and values it reads)"""
        return [(i, part, j) for i, l in enumerate(self.layers) if isinstance(l.mixer, SumMixer)
                for part, j in l.mixer.kv_sources().items()]

    def _check_kv_sources(self) -> None:
        for i, part, j in self._kv_sources():
            if self.cfg.loop:
                raise ValueError("layers that read another's keys and values do not run in loops")
            source = self.layers[j].mixer if 0 <= j < i else None
            if not isinstance(source, SumMixer) or part not in source.parts or not self.layers[i].mixer.parts[part].reads(
                    source.parts[part]):
                raise ValueError(f"layer {i} reads the keys and values of layer {j}: an earlier layer with projections of its "
                                 "own, the same sizes and rotation is needed")

    # ---- runtime ---------------------------------------------------------------------------------------
    def setup_runtime(self, max_tokens: int, tw_cfg, provider: Optional[str] = None,
                      disable_custom_all_reduce: bool = True) -> HybridRuntime:
        self.rt = HybridRuntime(self.cfg, max_tokens, self.final_norm_w.device, tw_cfg, provider)
        for layer in self.layers:
            m = layer.mixer
            for part in (m, layer.mlp):
                for name, cols in part.workspaces() if part is not None else ():
                    self.rt.buffer(name, max_tokens, cols)
                if self.tiles and part is m and isinstance(m, LatentAttention):
                    for name, cols in m.context_workspaces():
                        self.rt.buffer(name, self.rt.context_rows, cols)
            m.bind_runtime(self.rt)
            if layer.mlp is not None:
                layer.mlp.bind_runtime(self.rt)
        return self.rt

    def kv_cache_bytes_per_block(self, block_size: int) -> int:
        return max(1, sum(self.layers[i].mixer.cache_bytes_per_block(block_size) for i, _ in self.runs))

    def state_bytes_per_slot(self) -> int:
        return sum(self.layers[i].mixer.state_bytes_per_slot() for i, _ in self.runs)

    def init_kv_cache(self, num_blocks: int, block_size: int) -> None:
        for (i, _), kept in zip(self.runs, self.kept):
            self.layers[i].mixer.init_cache(kept, num_blocks, block_size)
        for i, part, j in self._kv_sources():
            self.layers[i].mixer.share_cache(part, self.kept[i], self.kept[j])

    def init_state(self, num_slots: int) -> None:
        for (i, _), kept in zip(self.runs, self.kept):
            self.layers[i].mixer.init_state(kept, num_slots)

    def cache_tensors(self) -> list[torch.Tensor]:
        return list({id(t): t for kept in self.kept for t in _tensors(kept)}.values())      # (some are shared)

    def drop_caches(self) -> None:
        self.kept = [self.layers[i].mixer.new_kept() for i, _ in self.runs]

    # ---- a step's layout -------------------------------------------------------------------------------
    def plan_step(self, q_lens, kv_lens, state_slots, prev_tokens):
        """Routing of a step's rows: (attention plan as of ``plan_attention``, extra int32 arrays, host values).
        ``prev_tokens``: the token before each sequence's first row of the step, -1 where there is none.

        Attention: a run of a prompt goes to 128-query tiles. In models with latent attention it does so when it is long
        enough to pay for expanding its context (a product over the whole context, whatever the run's length), and when
        the context fits the workspace. Every other row is attended alone (over latents: in the absorbed form).
        Recurrences: long runs in chunks, short ones token by token."""
        B = len(q_lens)
        extra = {"prev_token": np.asarray(prev_tokens, dtype=np.int32)} if self.bigram_w is not None else {}
        if max(q_lens) == 1:
            rows = np.arange(B, dtype=np.int32)
            plan = ([], [], rows, rows, np.asarray(kv_lens, dtype=np.int32))
            extra["row_seq"] = rows
            if self.recurrent:
                extra.update(state_slots=np.asarray(state_slots, dtype=np.int32), scan_seqs=rows, chunk_seqs=rows[:0])
            return plan, extra, {}
        n = np.asarray(q_lens)
        tiled, ctx_rows, first = [], 0, {}
        if self.tiles and not self.expand:
            tiled = [b for b, ql in enumerate(q_lens) if ql >= PREFILL_MIN_Q]
        elif self.tiles:
            for b, (ql, kv) in enumerate(zip(q_lens, kv_lens)):
                # whole key tiles from the first visible key's on
                lo = max(0, kv - ql - self.expand_window + 1) // 128 * 128 if self.expand_window else 0
                rows = kv - lo
                if (ql >= 64 or (ql >= PREFILL_MIN_Q and rows <= 2 * ql)) and ctx_rows + rows <= self.rt.context_rows:
                    tiled.append(b)
                    first[b] = lo
                    ctx_rows += rows
        row_seq = np.repeat(np.arange(B, dtype=np.int32), n)
        start = np.cumsum(n) - n
        tok_row = np.flatnonzero(~np.isin(row_seq, tiled)).astype(np.int32)
        tok_seq = row_seq[tok_row]
        tok_kv = (np.asarray(kv_lens) - n)[tok_seq] + (tok_row - start[tok_seq]) + 1
        tile_seq = [b for b in tiled for _ in range(0, q_lens[b], 128)]
        tile_q0 = [q0 for b in tiled for q0 in range(0, q_lens[b], 128)]
        order = np.argsort([-(kv_lens[b] - q_lens[b] + q0) for b, q0 in zip(tile_seq, tile_q0)], kind="stable")
        plan = ([tile_seq[i] for i in order], [tile_q0[i] for i in order], tok_row, tok_seq, tok_kv.astype(np.int32))
        host = {}
        extra["row_seq"] = row_seq
        if tiled and self.expand:
            cu = np.zeros(len(tiled) + 1, dtype=np.int32)
            lo = np.asarray([first[b] for b in tiled], dtype=np.int32)
            np.cumsum([kv_lens[b] - first[b] for b in tiled], out=cu[1:])
            begin = np.full(B, -1, dtype=np.int32)
            begin[tiled] = cu[:-1] - lo              # the workspace row of key 0, were it there
            extra.update(ctx_seqs=np.asarray(tiled, dtype=np.int32), ctx_cu=cu, ctx_begin=begin, ctx_first=lo)
            host = {"ctx_rows": int(cu[-1]), "ctx_max": max(kv_lens[b] - first[b] for b in tiled)}
        if self.recurrent:
            long = n >= hops.CHUNK_MIN_TOKENS
            extra.update(state_slots=np.asarray(state_slots, dtype=np.int32),
                         scan_seqs=np.flatnonzero(~long).astype(np.int32), chunk_seqs=np.flatnonzero(long).astype(np.int32))
        return plan, extra, host

    def launch_key(self, meta: AttentionMetadata, block_size: int) -> tuple:
        """What shapes a step's launches besides its token and sequence counts (part of a graph's signature)."""
        return (meta.all_single, tuple(sorted(meta.extra_cpu.items())),
                tuple(sorted((k, v.shape[0]) for k, v in meta.extra.items())),
                tuple(l.mixer.launch_key(meta, block_size, self.rt.sm_count) for l in self.layers))

    # ---- forward ---------------------------------------------------------------------------------------
    @torch.inference_mode()
    def forward(self, step) -> torch.Tensor:
        """Runs the stack; returns the final-norm rows ``[T, padded width]``."""
        rt, cfg, meta = self.rt, self.cfg, step.meta
        T, eps = step.plan.num_tokens, cfg.rms_norm_eps
        x32, xa, y = rt.residual[:T], rt.hidden[:T], rt.sublayer[:T]
        if cfg.block == "streams":
            self._forward_streams(step, x32.view(T, max(1, cfg.streams), -1), xa, y)
            return xa
        if cfg.block == "sandwich":
            self._forward_sandwich(step, x32, xa, y)
            return xa
        if cfg.block == "parallel":
            first = rt.first[:T] if rt.first is not None else None
            hops.embed_norm(step.input_ids, self.embed_w, self.bigram_w, cfg.bigram, meta, x32, first,
                            self.layers[self.runs[0][0]].norm1_w, eps, xa)
            for n, (i, _) in enumerate(self.runs):
                self.layers[i].mixer(xa, meta, rt, y, self.kept[n])
                nxt, again = self.runs[n + 1] if n + 1 < len(self.runs) else (None, False)
                hops.add_prenorm_(y, x32, first if again else None,
                                  self.final_norm_w if nxt is None else self.layers[nxt].norm1_w, eps, xa)
            return xa
        hops.embed_residual(step.input_ids, self.embed_w, x32, xa, cfg.hidden_size)
        last = self.layers[-1]
        for layer, kept in zip(self.layers, self.kept):
            layer.mixer(xa, meta, rt, y, kept)
            final = self.final_norm_w if layer is last and layer.mlp is None else None
            hops.postnorm_add_(y, x32, layer.norm1_w, eps, xa, final)
            if layer.mlp is not None:
                layer.mlp(xa, rt, y)
                hops.postnorm_add_(y, x32, layer.norm2_w, eps, xa, self.final_norm_w if layer is last else None)
        return xa

    def _forward_streams(self, step, x: torch.Tensor, xa: torch.Tensor, y: torch.Tensor) -> None:
        rt, cfg, meta = self.rt, self.cfg, step.meta
        eps, off = cfg.rms_norm_eps, cfg.norm_offset
        first = self.layers[0]
        hops.embed_streams(step.input_ids, self.embed_w, x, first.hc[0]["in"], first.norm1_w, off, eps, xa)
        for n, (layer, kept) in enumerate(zip(self.layers, self.kept)):
            nxt = self.layers[n + 1] if n + 1 < len(self.layers) else None
            behind = (None, self.final_norm_w) if nxt is None else (nxt.hc[0]["in"], nxt.norm1_w)
            layer.mixer(xa, meta, rt, y, kept)
            alike = n == 0                  # the streams, until the first sublayer
            if layer.mlp is not None:
                hops.streams_step(y, x, layer.hc[0], cfg.residual_mult, layer.hc[1]["in"], layer.norm2_w, off, eps, xa, alike)
                layer.mlp(xa, rt, y)
                alike = False
            hops.streams_step(y, x, layer.hc[-1], cfg.residual_mult, *behind, off, eps, xa, alike)

    def _forward_sandwich(self, step, x32: torch.Tensor, xa: torch.Tensor, y: torch.Tensor) -> None:
        rt, cfg, meta, eps = self.rt, self.cfg, step.meta, self.cfg.rms_norm_eps
        results = rt.results[:, :x32.shape[0]] if rt.results is not None else None
        hops.embed_sandwich(step.input_ids, self.embed_w, cfg.embed_scale, x32, results[0] if results is not None else None,
                            self.layers[0].norms["norm1"].pair, eps, xa)
        for i, (layer, kept) in enumerate(zip(self.layers, self.kept)):
            last = i + 1 == len(self.layers)
            nxt = (self.final_norm_w, self.final_norm_b) if last else self.layers[i + 1].norms["norm1"].pair
            norms = layer.norms
            layer.mixer(xa, meta, rt, y, kept)
            behind = norms["norm1b"]
            if layer.mlp is not None:
                hops.sandwich_step(y, x32, behind.pair, norms["norm2"].pair, eps, xa)
                layer.mlp(xa, rt, y)
                behind = norms["norm2b"]
            hops.sandwich_step(y, x32, behind.pair, nxt, eps, xa, layer.dwa, results, last)

    @torch.inference_mode()
    def compute_logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """fp32 logits ``[rows, vocab]``."""
        return self.head(hidden_rows)[:, : self.cfg.vocab_size].float() * self.cfg.logit_scale

    # ---- weights ---------------------------------------------------------------------------------------
    def tensor_targets(self) -> dict:
        V, W = self.cfg.vocab_size, self.cfg.hidden_size
        out = {"embed": ((V, W), lambda t: self.embed_w.data[:, :W].copy_(t)),
               "final.norm": ((W,), self.final_norm_w.data.copy_)}
        if self.final_norm_b is not None:
            out["final.norm.b"] = ((W,), self.final_norm_b.data.copy_)
        if not self.cfg.tie_word_embeddings:
            out["head"] = ((V, W), lambda t: self.head.load_rows(t, 0))
        if self.bigram_w is not None:
            out["bigram"] = ((self.bigram_w.shape[0], W), lambda t: self.bigram_w.data[:, :W].copy_(t))
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
            if name.endswith(("norm1", "norm2", "norm1b", "norm2b", "final.norm")):
                return t.fill_(1.0 - self.cfg.norm_offset)
            if name.endswith("norm") or leaf == "D":
                return t.fill_(1.0)
            if ".hc" in name:
                return t.copy_(torch.eye(shape[0]) if leaf.endswith("mix") else torch.full(shape, 1.0 / shape[0]))
            if leaf == "sink" or name.endswith(".correction"):
                return t.zero_()
            if leaf == "pb":                    # keys count about one in a few tens
                return t.fill_(-3.0)
            if leaf == "z.b":                   # memories of a few to a few hundred tokens
                return t.uniform_(-6.0, -1.0, generator=g)
            if name.endswith(".dwa"):
                t.fill_(0.2 / max(1, shape[0] - 1))
                t[-1] = 0.8
                return t
            if leaf == "A_log":
                return t.uniform_(1.0, 16.0, generator=g).log_()
            if leaf == "dt_bias":
                return t.uniform_(-6.9, -2.3, generator=g)
            if name.endswith(".b"):
                return t.zero_()
            if leaf.endswith("conv"):
                return t.normal_(0.0, shape[1] ** -0.5, generator=g)
            if name.endswith(".mlp.act"):
                return torch.tensor([1 / 3, 1 / 3, 1 / 3, 0.0], device=dev)
            return t.normal_(0.0, self.cfg.init_std, generator=g)
        for name, (shape, put) in self.tensor_targets().items():
            put(fill(name, shape))

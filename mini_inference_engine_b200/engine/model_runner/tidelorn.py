"""The Tidelorn decoder on the paged step machinery.

A post-norm decoder with a 32-bit residual stream: scaled token embedding + hashed bigram embedding + sinusoid;
per layer an attention mixer without rotation (query / key heads divided by their RMS, values blended with those
of the first value-mixing layer, a sink in the softmax) and a clamped gated feed-forward, each followed by an RMS
norm of ``alpha * x + sublayer(x)``.  Layers of type ``attention`` see the whole prefix, have projection biases, a
position-dependent query temperature and a learned sink per head; layers of type ``attention_2`` see a sliding
window and add one to the denominator.

Cache: per layer a key pool ``[pages, kv_heads, page, dim]`` and a value pool ``[pages, kv_heads, page, vdim]``
(layers may differ in every size), plus one pool of token ids ``[pages, page]`` that carries the previous token of
a sequence for the bigram embedding; all under the same block tables, so whatever moves, shares or frees a page
moves that state with it.  One layer is

  merged qkv projection -> norm / temperature / value mix / page write -> paged attention -> o projection ->
  scaled residual sum + norm -> merged gate_up projection -> clamped gate -> down projection ->
  scaled residual sum + norm
"""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from ..kernels.decoder_glue import clamped_glu, embed_tokens, qkv_norm_mix_write, sinusoid_turns, sum_rms_norm
from ..kv_cache.sink_attention import (
    attention_rows,
    sink_decode_attention,
    sink_decode_supported,
    sink_prefill_attention,
    sink_prefill_supported,
)
from ..kv_cache.triton_paged_attention import decode_scratch
from ... import _lib
from .step_runner import PLAN_SLOTS, PagedStepRunner

SINUSOID_BASE = 10000.0
GATE_SLOPE = 1.702
UP_OFFSET = 1.0
NORM_WEIGHT_OFFSET = 1.0  # norm weights are stored as their deviation from one


@dataclass(frozen=True)
class TidelornLayer:
    """Sizes and branches of one layer."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias: bool                              # biases in the q / k / v projections
    learned_sink: bool                      # a stored sink per head; otherwise a sink whose score is 0
    temperature: tuple[float, int] | None   # (coefficient, period)
    window: int | None
    v_mix: bool
    ff: int | None                          # None: no feed-forward (and no second norm)
    limit: float

    @property
    def qkv_rows(self) -> int:
        return (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim


@dataclass(frozen=True)
class TidelornShape:
    vocab: int
    width: int
    eps: float
    alpha: float
    embed_scale: float
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: tuple[TidelornLayer, ...]
    page: int = 16

    @property
    def first_v_mix(self) -> int | None:
        """Index of the layer whose values the later value-mixing layers blend in."""

        return next((i for i, layer in enumerate(self.layers) if layer.v_mix), None)

    @classmethod
    def from_config(cls, config: dict, page: int = 16) -> "TidelornShape":
        layers = []
        for index, entry in enumerate(config["layers"]):
            kind, mixer, mlp = entry["type"], entry["mixer"], entry.get("mlp")
            if kind not in ("attention", "attention_2"):
                raise ValueError(f"layer {index}: unknown type {kind!r}")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {index}: unknown feed-forward {mlp['kind']!r}")
            full = kind == "attention"
            temperature = None
            if full:
                temperature = (float(mixer["q_temp"]["coef"]), int(mixer["q_temp"]["every"]))
                if temperature[1] < 1:
                    raise ValueError(f"layer {index}: the temperature period must be positive")
            window = None if full else int(mixer["mask"]["size"])
            layer = TidelornLayer(
                heads=int(mixer["heads"]), kv_heads=int(mixer["kv_heads"]), dim=int(mixer["dim"]),
                vdim=int(mixer["vdim"]), scale=float(mixer["scale"]), bias=full, learned_sink=full,
                temperature=temperature, window=window, v_mix=bool(mixer.get("v_mix", False)),
                ff=None if mlp is None else int(mlp["ff"]), limit=0.0 if mlp is None else float(mlp["limit"]))
            if layer.heads < 1 or layer.kv_heads < 1 or layer.heads % layer.kv_heads:
                raise ValueError(f"layer {index}: query heads must be a multiple of key/value heads")
            if window is not None and window < 1:
                raise ValueError(f"layer {index}: the window must be positive")
            layers.append(layer)
        bigram = config["embedding"]["bigram"]
        shape = cls(vocab=int(config["vocab"]), width=int(config["width"]), eps=float(config["norm"]["eps"]),
                    alpha=float(config["postln_alpha"]), embed_scale=float(config["embedding"]["scale"]),
                    buckets=int(bigram["buckets"]), mul_prev=int(bigram["mul_prev"]), mul_cur=int(bigram["mul_cur"]),
                    layers=tuple(layers), page=page)
        sizes = {layer.kv_heads * layer.vdim for layer in layers if layer.v_mix}
        if len(sizes) > 1:
            raise ValueError("layers that mix values must agree in kv_heads * vdim")
        return shape

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Name and shape of every tensor of a checkpoint."""

        out = {"embed": (self.vocab, self.width), "bigram": (self.buckets + 1, self.width)}
        for i, layer in enumerate(self.layers):
            out[f"l{i}.norm1"] = (self.width,)
            if layer.ff is not None:
                out[f"l{i}.norm2"] = (self.width,)
            rows = {"q": layer.heads * layer.dim, "k": layer.kv_heads * layer.dim, "v": layer.kv_heads * layer.vdim}
            for name, n in rows.items():
                out[f"l{i}.mix.{name}"] = (n, self.width)
                if layer.bias:
                    out[f"l{i}.mix.{name}.b"] = (n,)
            if layer.v_mix:
                out[f"l{i}.mix.vmix"] = ()
            if layer.learned_sink:
                out[f"l{i}.mix.sink"] = (layer.heads,)
            out[f"l{i}.mix.o"] = (self.width, layer.heads * layer.vdim)
            if layer.ff is not None:
                out[f"l{i}.mlp.gate"] = out[f"l{i}.mlp.up"] = (layer.ff, self.width)
                out[f"l{i}.mlp.down"] = (self.width, layer.ff)
        out["final.norm"] = (self.width,)
        out["head"] = (self.vocab, self.width)
        return out


@dataclass
class TidelornLayerWeights:
    qkv: torch.Tensor
    qkv_bias: torch.Tensor | None
    o: torch.Tensor
    sinks: torch.Tensor              # fp32, one per query head
    lam: float                       # weight of the first mixing layer's values; 0 where nothing is blended in
    norm1: torch.Tensor
    gate_up: torch.Tensor | None
    down: torch.Tensor | None
    norm2: torch.Tensor | None


class TidelornWeights:
    """Weights in the form the runner uses: q / k / v and gate / up merged, everything in ``dtype`` except the
    sinks (fp32) and the value-mixing factors (host numbers)."""

    def __init__(self, shape: TidelornShape, take, device: torch.device, dtype: torch.dtype = torch.bfloat16) -> None:
        """``take(name, shape)`` returns a checkpoint tensor."""

        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("weights are bfloat16 or float32")
        self.shape, self.device, self.dtype = shape, device, dtype
        shapes = shape.tensor_shapes()

        def fetch(name: str) -> torch.Tensor:
            return take(name, shapes[name]).to(device=device, dtype=dtype).contiguous()

        self.embed, self.bigram = fetch("embed"), fetch("bigram")
        self.layers: list[TidelornLayerWeights] = []
        for i, layer in enumerate(shape.layers):
            mix = f"l{i}.mix."
            qkv = torch.cat([fetch(mix + n) for n in "qkv"])
            bias = torch.cat([fetch(mix + n + ".b") for n in "qkv"]) if layer.bias else None
            lam = float(take(mix + "vmix", ()).float()) if layer.v_mix else 0.0
            if i == shape.first_v_mix:
                lam = 0.0
            sinks = (take(mix + "sink", shapes[mix + "sink"]).to(device=device, dtype=torch.float32).contiguous()
                     if layer.learned_sink else torch.zeros(layer.heads, dtype=torch.float32, device=device))
            dense = layer.ff is not None
            self.layers.append(TidelornLayerWeights(
                qkv, bias, fetch(mix + "o"), sinks, lam, fetch(f"l{i}.norm1"),
                torch.cat([fetch(f"l{i}.mlp.gate"), fetch(f"l{i}.mlp.up")]) if dense else None,
                fetch(f"l{i}.mlp.down") if dense else None, fetch(f"l{i}.norm2") if dense else None))
        self.final_norm, self.head = fetch("final.norm"), fetch("head")
        self.turns = sinusoid_turns(shape.width, SINUSOID_BASE, device)

    @classmethod
    def random(cls, shape: TidelornShape, device: torch.device, *, seed: int = 0,
               dtype: torch.dtype = torch.bfloat16) -> "TidelornWeights":
        """Seeded random weights of the checkpoint's form (drawn on ``device``)."""

        generator = torch.Generator(device=device).manual_seed(seed)

        def take(name: str, size: tuple[int, ...]) -> torch.Tensor:
            noise = torch.randn(size, generator=generator, device=device, dtype=torch.float32)
            if name.endswith("vmix"):
                noise = noise.mul(0.1).add(0.5)
            elif "norm" in name:
                noise = noise * 0.1
            elif name.endswith((".b", "sink")):
                noise = noise * 0.5
            elif name not in ("embed", "bigram"):
                noise = noise / math.sqrt(size[1])
            return noise.to(torch.bfloat16)

        return cls(shape, take, device, dtype)

    def weight_bytes(self) -> int:
        """Bytes a decode step streams (projections, feed-forward and head; the embedding rows are a few)."""

        total = self.head.numel()
        for layer in self.layers:
            total += sum(t.numel() for t in (layer.qkv, layer.o, layer.gate_up, layer.down) if t is not None)
        return total * self.dtype.itemsize


class TidelornRunner(PagedStepRunner):
    """Steps of a Tidelorn model over its paged cache (pages, buckets and graphs: ``PagedStepRunner``)."""

    def __init__(self, weights: TidelornWeights, *, num_pages: int, max_batch: int, max_context: int,
                 decode_buckets: tuple[int, ...] | None = None, chunk_buckets: tuple[int, ...] = (128, 512),
                 max_chunks: int = 4, kv_init: str = "zeros", attention: str = "auto") -> None:
        """``attention``: "auto" takes the streaming kernels where a layer's sizes and number format allow them,
        "rows" the row kernel everywhere."""

        if attention not in ("auto", "rows"):
            raise ValueError("attention must be 'auto' or 'rows'")
        super().__init__(weights.shape, weights.device, num_pages=num_pages, max_batch=max_batch,
                         max_context=max_context, decode_buckets=decode_buckets, chunk_buckets=chunk_buckets,
                         max_chunks=max_chunks)
        self.weights, self.dtype = weights, weights.dtype
        # Library products accumulate in full fp32: no TF32 for fp32 operands, no bf16 partial sums for bf16 ones.
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        self.key_blocks, self.value_blocks = [], []
        for layer in self.shape.layers:
            for pool, size in ((self.key_blocks, layer.dim), (self.value_blocks, layer.vdim)):
                blocks = torch.zeros(self.total_pages, layer.kv_heads, self.shape.page, size, dtype=self.dtype,
                                     device=self.device)
                if kv_init == "normal":
                    blocks.normal_()
                pool.append(blocks)
        # Layers of one geometry share a split-KV work plan within a step, and its scratch: (scratch key, streams
        # decode rows, streams chunks) per layer.
        self._attention: list[tuple[tuple, bool, bool]] = []
        self._scratch: dict[tuple, torch.Tensor] = {}
        rows = max(max_batch, self.decode_buckets[-1])
        for layer in self.shape.layers:
            sizes = (layer.dim, layer.vdim, self.shape.page, self.dtype)
            decode = attention == "auto" and sink_decode_supported(*sizes)
            chunks = attention == "auto" and sink_prefill_supported(layer.heads, layer.kv_heads, *sizes, layer.scale)
            key = (layer.heads, layer.kv_heads, layer.dim, layer.vdim, layer.window)
            if decode and key not in self._scratch:
                reach = max_context if layer.window is None else min(max_context, layer.window + 16)
                self._scratch[key] = decode_scratch(rows, layer.heads, layer.kv_heads, layer.vdim, rows * reach,
                                                    self.device)
            self._attention.append((key, decode, chunks))
        self.history = torch.zeros(self.total_pages, self.shape.page, dtype=torch.int32, device=self.device)

    # -- projections ----------------------------------------------------------------------------

    @staticmethod
    def _linear(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor | None = None) -> torch.Tensor:
        return torch.nn.functional.linear(x, weight, bias)

    def _logits(self, final: torch.Tensor) -> torch.Tensor:
        """fp32 logits of normed rows."""

        head = self.weights.head.t()
        return torch.mm(final, head) if self.dtype == torch.float32 else torch.mm(final, head, out_dtype=torch.float32)

    def _finish(self, x32: torch.Tensor, return_logits: bool):
        """Final norm, then greedy tokens (and the logits when asked for) of residual rows."""

        _, final = sum_rms_norm(x32, None, self.weights.final_norm, eps=self.shape.eps,
                                weight_offset=NORM_WEIGHT_OFFSET, keep32=False)
        if not return_logits and self.can_fuse_lm_head(final, self.weights.head):
            return self.lm_head_argmax(final, self.weights.head)
        logits = self._logits(final)
        tokens = logits.argmax(dim=-1)
        return (tokens, logits) if return_logits else tokens

    # -- the layers -----------------------------------------------------------------------------

    def _attend(self, index: int, queries: torch.Tensor, attended: torch.Tensor, positions, token_to_sequence,
                block_tables, plans: dict, *, decode_rows: int, decode_lengths, cu_seqlens=None, kv_lens=None,
                max_query_len: int = 0) -> None:
        """Attention of one layer: the leading ``decode_rows`` rows, then the packed chunks.  ``plans`` counts the
        layers that have used each work plan of this step."""

        layer, sinks = self.shape.layers[index], self.weights.layers[index].sinks
        keys, values = self.key_blocks[index], self.value_blocks[index]
        common = dict(scale=layer.scale, window=layer.window, sinks=sinks, status=self.status)
        key, stream_decode, stream_chunks = self._attention[index]
        parts = []  # row ranges left to the row kernel
        if decode_rows and stream_decode:
            used = plans.get(key, 0)
            plans[key] = used + 1
            sink_decode_attention(queries[:decode_rows], attended[:decode_rows], keys, values,
                                  block_tables[:decode_rows], decode_lengths, scratch=self._scratch[key],
                                  use_plan=used % PLAN_SLOTS != 0, plan_slot=used % PLAN_SLOTS, **common)
        elif decode_rows:
            parts.append(slice(0, decode_rows))
        if queries.shape[0] > decode_rows:
            if stream_chunks:
                sink_prefill_attention(queries[decode_rows:], attended[decode_rows:], keys, values,
                                       block_tables[decode_rows:], cu_seqlens, kv_lens, max_query_len=max_query_len,
                                       **common)
            else:
                parts.append(slice(decode_rows, queries.shape[0]))
        for rows in parts:
            attention_rows(queries[rows], attended[rows], keys, values, positions[rows],
                           None if token_to_sequence is None else token_to_sequence[rows], block_tables, **common)

    def _layers(self, input_ids, positions, token_to_sequence, block_tables, **batch) -> torch.Tensor:
        """Residual rows after the last layer (fp32), the cache holding the new tokens."""

        shape, weights = self.shape, self.weights
        tokens = int(input_ids.shape[0])
        x32, x = embed_tokens(input_ids, weights.embed, positions, token_to_sequence, block_tables,
                              scale=shape.embed_scale, page=shape.page, num_pages=self.total_pages,
                              bigram=weights.bigram, mul_prev=shape.mul_prev, mul_cur=shape.mul_cur,
                              history=self.history, turns=weights.turns, status=self.status)
        v_first, plans = None, {}
        norm = dict(eps=shape.eps, alpha=shape.alpha, weight_offset=NORM_WEIGHT_OFFSET)
        for index, (layer, w) in enumerate(zip(shape.layers, weights.layers)):
            qkv = self._linear(x, w.qkv, w.qkv_bias)
            queries = torch.empty(tokens, layer.heads, layer.dim, dtype=self.dtype, device=self.device)
            qkv_norm_mix_write(qkv, queries, self.key_blocks[index], self.value_blocks[index], positions,
                               token_to_sequence, block_tables, q_heads=layer.heads, kv_heads=layer.kv_heads,
                               dim=layer.dim, value_dim=layer.vdim, unit_norm=True, eps=shape.eps,
                               temperature=layer.temperature, lam=w.lam,
                               v_first=v_first if layer.v_mix else None, status=self.status)
            if index == shape.first_v_mix:
                v_first = qkv[:, (layer.heads + layer.kv_heads) * layer.dim:]
            attended = torch.empty(tokens, layer.heads, layer.vdim, dtype=self.dtype, device=self.device)
            self._attend(index, queries, attended, positions, token_to_sequence, block_tables, plans, **batch)
            mixed = self._linear(attended.view(tokens, layer.heads * layer.vdim), w.o)
            x32, x = sum_rms_norm(x32, mixed, w.norm1, **norm)
            if layer.ff is not None:
                act = clamped_glu(self._linear(x, w.gate_up), limit=layer.limit, slope=GATE_SLOPE, up_offset=UP_OFFSET)
                x32, x = sum_rms_norm(x32, self._linear(act, w.down), w.norm2, **norm)
        return x32

    # -- the two forwards -----------------------------------------------------------------------

    def decode_forward(self, input_ids: torch.Tensor, sequence_lengths: torch.Tensor, block_tables: torch.Tensor,
                       return_logits: bool = False):
        """One token per block-table row, at position ``length - 1`` (``sequence_lengths`` counts it).  Returns
        the greedy next tokens (int64), with ``return_logits`` also their fp32 logits."""

        before = _lib.load().mie_launch_count()
        batch = int(input_ids.shape[0])
        x32 = self._layers(input_ids, sequence_lengths - 1, None, block_tables, decode_rows=batch,
                           decode_lengths=sequence_lengths)
        out = self._finish(x32, return_logits)
        self.launches_per_step = int(_lib.load().mie_launch_count() - before)
        return out

    def mixed_forward(self, input_ids: torch.Tensor, token_to_sequence: torch.Tensor, token_positions: torch.Tensor,
                      block_tables: torch.Tensor, *, decode_rows: int, decode_lengths, cu_seqlens: torch.Tensor,
                      kv_lens: torch.Tensor, max_query_len: int, logit_rows: torch.Tensor,
                      return_logits: bool = False):
        """Decode rows (one per leading block-table row) and packed prompt chunks in one flat stream; the rows in
        ``logit_rows`` are projected to logits."""

        before = _lib.load().mie_launch_count()
        x32 = self._layers(input_ids, token_positions, token_to_sequence, block_tables, decode_rows=decode_rows,
                           decode_lengths=decode_lengths, cu_seqlens=cu_seqlens, kv_lens=kv_lens,
                           max_query_len=max_query_len)
        out = self._finish(x32.index_select(0, logit_rows), return_logits)
        self.launches_per_step = int(_lib.load().mie_launch_count() - before)
        return out


__all__ = ["TidelornLayer", "TidelornRunner", "TidelornShape", "TidelornWeights"]

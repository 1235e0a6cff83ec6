"""Flat-token Qwen3 forward over the sm_100a kernels, with a CUDA-graph decode step.

Takes the place of the captured decode forward of the reference
(engine/serving/chunked_prefill.py:206-298: ``_graph_decode_call`` /
``_capture_decode_graph`` / ``_decode``) and of the flat layer loops
(engine/model_runner/qwen3_mixed.py:125, qwen3_packed.py:29).  The reference
drives Hugging Face's ``Qwen3ForCausalLM`` and monkey-patches its modules; this
runner owns plain weight tensors and calls the kernels directly, so one decode
layer is a dozen launches of this library's kernels:

  add+RMSNorm(+quant) -> FP8 GEMM (merged qkv) -> q/k-norm + RoPE + KV write ->
  paged decode attention -> quant -> FP8 GEMM (o) [all-reduce] ->
  add+RMSNorm(+quant) -> FP8 GEMM (merged gate_up) -> SiLU*up(+quant) ->
  FP8 GEMM (down) [all-reduce]

Tensor parallelism is by heads: rank r of t owns query heads [32r/t, 32(r+1)/t)
and KV heads [8r/t, 8(r+1)/t) with its own K/V page pool, the merged qkv and
gate_up projections are column-parallel, o and down are row-parallel.  Their
partial sums are combined by ``mie_tp_reduce_rms_norm`` (one kernel per rank
over IPC-mapped peer memory that also does the residual add, the RMSNorm and
the FP8 quantisation for the next GEMM; ``MIE_TP_EXCHANGE=nccl`` selects a
plain NCCL all-reduce instead).  The tied lm_head is vocabulary-sharded and
greedy sampling exchanges one (value, index) pair per row over NCCL.  The
library is reached through its C-ABI with ``ctypes``; PyTorch owns tensors,
streams and CUDA graphs only.
"""

from __future__ import annotations

import math
import os
from dataclasses import dataclass

import torch

from ... import _lib
from ..kernels import sm89_fp8
from .peer_exchange import PeerExchange
from .step_runner import (
    DEFAULT_DECODE_BUCKETS,
    PADDING,
    PLAN_SLOTS,
    DecodeBuffers,
    MixedBuffers,
    PagedStepRunner,
    select_bucket,
)
from ..kv_cache.fp8_kv import Fp8KvPool, launch_decode_attention_kv8
from ..kv_cache.triton_flash_prefill import launch_flash_prefill
from ..kv_cache.triton_paged_attention import decode_scratch, launch_decode_attention


@dataclass(frozen=True)
class Qwen3Shape:
    """Architecture constants (defaults: Qwen3-4B)."""

    layers: int = 36
    hidden: int = 2560
    q_heads: int = 32
    kv_heads: int = 8
    head_dim: int = 128
    intermediate: int = 9728
    vocab: int = 151936
    rms_eps: float = 1e-6
    rope_theta: float = 5_000_000.0
    page: int = 16


def quantize_weight_blocks(weight: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """e4m3 weight + one fp32 scale per 128x128 block (``amax / 448``), on the weight's device."""

    n, k = weight.shape
    nb, kb = -(-n // 128), -(-k // 128)
    padded = torch.zeros(nb * 128, kb * 128, dtype=torch.float32, device=weight.device)
    padded[:n, :k] = weight.float()
    blocks = padded.view(nb, 128, kb, 128)
    scales = blocks.abs().amax(dim=(1, 3)) / 448.0
    quantized = (blocks / scales.clamp_min(1e-12)[:, None, :, None]).view(nb * 128, kb * 128)[:n, :k]
    return quantized.to(torch.float8_e4m3fn).contiguous(), scales.contiguous()


@dataclass
class LayerWeights:
    qkv: torch.Tensor
    qkv_scale: torch.Tensor
    o: torch.Tensor
    o_scale: torch.Tensor
    gate_up: torch.Tensor
    gate_up_scale: torch.Tensor
    down: torch.Tensor
    down_scale: torch.Tensor
    input_norm: torch.Tensor
    post_norm: torch.Tensor
    q_norm: torch.Tensor
    k_norm: torch.Tensor


def shard_bounds(n: int, tp_size: int, tp_rank: int) -> tuple[int, int]:
    """Rows ``[start, stop)`` of an ``n``-row dimension that rank ``tp_rank`` of ``tp_size`` owns."""

    return n // tp_size * tp_rank, n // tp_size * (tp_rank + 1)


def scale_window(start: int, stop: int, block: int = 128) -> tuple[int, int]:
    """The smallest range of whole scale blocks ``[base, end)`` that covers ``[start, stop)``."""

    return start // block * block, -(-stop // block) * block


def _window_rows(w8: torch.Tensor, scales: torch.Tensor, start: int, stop: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Rows ``[start, stop)`` of a block-quantised ``[N, K]`` weight, placed inside their scale window: the
    result has ``end - base`` rows (zeros outside the shard) and the window's rows of the scale grid, so a
    shard that starts in the middle of a 128-row scale block keeps the unsharded block's scale."""

    base, end = scale_window(start, stop)
    out = torch.zeros(end - base, w8.shape[1], dtype=torch.uint8, device=w8.device)
    out[start - base:stop - base] = w8[start:stop].view(torch.uint8)
    rows = scales[base // 128:end // 128]
    if rows.shape[0] < (end - base) // 128:  # the window runs past the last (partial) block
        rows = torch.cat([rows, rows.new_zeros((end - base) // 128 - rows.shape[0], rows.shape[1])])
    return out.view(torch.float8_e4m3fn), rows.contiguous()


class Qwen3Weights:
    """Seeded random-init weights in the checkpoint's format, sharded for one tensor-parallel rank.

    Every rank draws the full tensors from the same per-layer seed, quantises them on the UNSHARDED
    128x128 block grid (what a checkpoint holds) and keeps its slice of the e4m3 values and of the scale
    grid, so all ranks of a group hold consistent shards and a shard is bit for bit a slice of the
    single-GPU model.  Head shards are whole scale blocks (head_dim 128).  An MLP shard need not be: at 8
    ranks 9728 / 8 = 1216 = 9.5 blocks, so odd ranks start 64 rows into a block.  Such a shard is stored
    inside its window of whole scale blocks (``inter_window`` wide, the shard at ``inter_offset``, zeros
    around it): gate and up each occupy one window of the merged gate_up weight, and down_proj's K
    dimension is the window, so every kernel keeps seeing 128-aligned scale blocks and the zero rows /
    columns contribute exact zeros.
    """

    def __init__(self, shape: Qwen3Shape, device: torch.device, *, seed: int = 0, tp_rank: int = 0,
                 tp_size: int = 1, layers: int | None = None) -> None:
        if shape.kv_heads % tp_size or shape.q_heads % tp_size or shape.vocab % tp_size:
            raise ValueError("tensor-parallel size must divide the head counts and the vocabulary")
        self.shape, self.device, self.tp_rank, self.tp_size = shape, device, tp_rank, tp_size
        d, hd = shape.hidden, shape.head_dim
        q_rows, kv_rows, inter = shape.q_heads * hd, shape.kv_heads * hd, shape.intermediate
        if inter % tp_size or (inter // tp_size) % 16:
            raise ValueError("tensor-parallel size must divide the MLP width into multiples of 16")
        if (q_rows // tp_size) % 128 or (kv_rows // tp_size) % 128:
            raise ValueError("a rank's query / KV head rows must be whole 128-row scale blocks")
        q_lo, q_hi = shard_bounds(q_rows, tp_size, tp_rank)
        kv_lo, kv_hi = shard_bounds(kv_rows, tp_size, tp_rank)
        i_lo, i_hi = shard_bounds(inter, tp_size, tp_rank)
        base, end = scale_window(i_lo, i_hi)
        self.inter_window, self.inter_offset, self.inter_width = end - base, i_lo - base, i_hi - i_lo

        def draw(generator: torch.Generator, rows: int, cols: int) -> torch.Tensor:
            return torch.randn(rows, cols, generator=generator, device=device, dtype=torch.float32) * 0.02

        def norm_weight(generator: torch.Generator, width: int) -> torch.Tensor:
            noise = torch.randn(width, generator=generator, device=device, dtype=torch.float32)
            return (1.0 + 0.1 * noise).to(torch.bfloat16)

        self.layers: list[LayerWeights] = []
        for index in range(shape.layers if layers is None else layers):
            generator = torch.Generator(device=device).manual_seed(seed * 100003 + index)
            wq, wk, wv = draw(generator, q_rows, d), draw(generator, kv_rows, d), draw(generator, kv_rows, d)
            wo = draw(generator, d, q_rows)
            wg, wu = draw(generator, inter, d), draw(generator, inter, d)
            wd = draw(generator, d, inter)
            (q8, q_s), (k8, k_s), (v8, v_s) = (quantize_weight_blocks(w) for w in (wq, wk, wv))
            o8, o_s = quantize_weight_blocks(wo)
            (g8, g_s), (u8, u_s) = quantize_weight_blocks(wg), quantize_weight_blocks(wu)
            d8, d_s = quantize_weight_blocks(wd)
            del wq, wk, wv, wo, wg, wu, wd
            qkv8 = torch.cat([q8[q_lo:q_hi], k8[kv_lo:kv_hi], v8[kv_lo:kv_hi]]).contiguous()
            qkv_s = torch.cat([q_s[q_lo // 128:q_hi // 128], k_s[kv_lo // 128:kv_hi // 128],
                               v_s[kv_lo // 128:kv_hi // 128]]).contiguous()
            o_local = o8[:, q_lo:q_hi].contiguous()
            o_local_s = o_s[:, q_lo // 128:q_hi // 128].contiguous()
            gate8, gate_s = _window_rows(g8, g_s, i_lo, i_hi)
            up8, up_s = _window_rows(u8, u_s, i_lo, i_hi)
            gu8, gu_s = torch.cat([gate8, up8]).contiguous(), torch.cat([gate_s, up_s]).contiguous()
            down8 = torch.zeros(d, end - base, dtype=torch.uint8, device=device)
            down8[:, i_lo - base:i_hi - base] = d8[:, i_lo:i_hi].view(torch.uint8)
            down_s = d_s[:, base // 128:end // 128]
            if down_s.shape[1] < (end - base) // 128:
                down_s = torch.cat([down_s, down_s.new_zeros(down_s.shape[0], (end - base) // 128 - down_s.shape[1])],
                                   dim=1)
            self.layers.append(LayerWeights(
                qkv8, qkv_s, o_local, o_local_s, gu8, gu_s, down8.view(torch.float8_e4m3fn), down_s.contiguous(),
                norm_weight(generator, d), norm_weight(generator, d),
                norm_weight(generator, hd), norm_weight(generator, hd),
            ))
            del q8, k8, v8, o8, g8, u8, d8
        generator = torch.Generator(device=device).manual_seed(seed * 100003 + 99991)
        self.embedding = (torch.randn(shape.vocab, d, generator=generator, device=device, dtype=torch.float32)
                          * 0.02).to(torch.bfloat16)
        self.final_norm = norm_weight(generator, d)
        # Tied lm_head, vocabulary-sharded: this rank scores rows [vocab_start, vocab_start + vocab / tp).
        v_lo, v_hi = shard_bounds(shape.vocab, tp_size, tp_rank)
        self.vocab_start = v_lo
        self.lm_head = self.embedding[v_lo:v_hi]

    def to(self, device: torch.device) -> "Qwen3Weights":
        """The same weights on another device (a CPU-drawn model is bit-identical on every host, a
        CUDA-drawn one follows the GPU's generator)."""

        import copy

        clone = copy.copy(self)
        clone.device = device
        clone.layers = [LayerWeights(*[getattr(layer, name).to(device) for name in layer.__dataclass_fields__])
                        for layer in self.layers]
        clone.embedding, clone.final_norm = self.embedding.to(device), self.final_norm.to(device)
        lo = self.vocab_start
        clone.lm_head = clone.embedding[lo:lo + self.lm_head.shape[0]]
        return clone

    def weight_bytes(self) -> int:
        total = self.lm_head.numel() * 2
        for layer in self.layers:
            for t in (layer.qkv, layer.o, layer.gate_up, layer.down):
                total += t.numel()
            for t in (layer.qkv_scale, layer.o_scale, layer.gate_up_scale, layer.down_scale):
                total += t.numel() * 4
        return total


def rope_table(shape: Qwen3Shape, max_positions: int, device: torch.device) -> torch.Tensor:
    """``[max_positions, 2, head_dim]`` bf16: cos row and sin row per position, built as HF's
    ``Qwen3RotaryEmbedding`` does (fp32 angles, cast at the end)."""

    inv_freq = 1.0 / (shape.rope_theta ** (torch.arange(0, shape.head_dim, 2, dtype=torch.int64,
                                                         device=device).float() / shape.head_dim))
    angles = torch.arange(max_positions, device=device, dtype=torch.float32).unsqueeze(1) * inv_freq
    emb = torch.cat((angles, angles), dim=-1)
    return torch.stack((emb.cos(), emb.sin()), dim=1).to(torch.bfloat16).contiguous()


def sharded_greedy_tokens(local_logits: torch.Tensor, vocab_start: int, tp_size: int, group=None) -> torch.Tensor:
    """Greedy token ids from vocabulary-sharded logits ``[batch, vocab / tp]``.

    Every rank contributes its best (value, global index) pair per row; one all-gather later each rank
    picks the pair with the largest value (lowest rank wins ties, which is also the lowest index).
    """

    batch = local_logits.shape[0]
    best_value, best_index = local_logits.float().max(dim=-1)
    if tp_size == 1:
        return best_index + vocab_start
    pair = torch.stack((best_value, (best_index + vocab_start).float()), dim=-1).contiguous()
    flat = torch.empty(tp_size * batch, 2, dtype=torch.float32, device=local_logits.device)
    torch.distributed.all_gather_into_tensor(flat, pair, group=group)
    gathered = flat.view(tp_size, batch, 2)
    winner = gathered[:, :, 0].argmax(dim=0)
    return gathered[winner, torch.arange(batch, device=local_logits.device), 1].long()


def sharded_greedy_from_pairs(tokens: torch.Tensor, values: torch.Tensor, tp_size: int, group=None) -> torch.Tensor:
    """Global greedy tokens from every rank's local winner: ``tokens`` are global vocabulary indices, ``values``
    order-preserving keys of the winning bf16 logits (``mie_lm_head_argmax``).  The largest value wins; among
    equal values the lowest rank, whose shard holds the lower indices."""

    if tp_size == 1:
        return tokens
    rows = tokens.shape[0]
    pair = torch.stack((values.long(), tokens), dim=-1).contiguous()
    flat = torch.empty(tp_size * rows, 2, dtype=torch.int64, device=tokens.device)
    torch.distributed.all_gather_into_tensor(flat, pair, group=group)
    gathered = flat.view(tp_size, rows, 2)
    winner = gathered[:, :, 0].argmax(dim=0)
    return gathered[winner, torch.arange(rows, device=tokens.device), 1]


class Qwen3DecodeRunner(PagedStepRunner):
    """Steps of a Qwen3-shaped FP8 model over paged KV (pages, buckets and graphs: ``PagedStepRunner``)."""

    def __init__(self, weights: Qwen3Weights, *, num_pages: int, max_batch: int, max_context: int,
                 process_group=None, kv_init: str = "zeros", fused_exchange: bool | None = None,
                 decode_buckets: tuple[int, ...] | None = None, chunk_buckets: tuple[int, ...] = (128, 512),
                 max_chunks: int = 4, kv_dtype: str = "bf16") -> None:
        super().__init__(weights.shape, weights.device, num_pages=num_pages, max_batch=max_batch,
                         max_context=max_context, decode_buckets=decode_buckets, chunk_buckets=chunk_buckets,
                         max_chunks=max_chunks)
        self.weights, self.group = weights, process_group
        self.tp = weights.tp_size
        shape = self.shape
        self.local_q_heads = shape.q_heads // self.tp
        self.local_kv_heads = shape.kv_heads // self.tp
        self.local_inter = weights.inter_window  # the MLP shard inside its window of whole scale blocks
        layers = len(weights.layers)
        if kv_dtype not in ("bf16", "fp8"):
            raise ValueError("kv_dtype must be 'bf16' or 'fp8'")
        self.kv_dtype = kv_dtype
        self.kv8 = None
        if kv_dtype == "fp8":
            # Opt-in e4m3 K/V pool (one fp32 scale per token and KV head).  Decode rows read it directly;
            # prompt chunks attend bf16 staging copies of their pages.  bf16 stays the default and the parity path.
            if shape.page != 16 or shape.head_dim != 128:
                raise ValueError("the FP8 KV cache needs 16-token pages and head_dim 128")
            self.kv8 = Fp8KvPool(layers, self.total_pages, self.local_kv_heads, self.device)
            self.key_blocks = self.value_blocks = None
            if kv_init == "normal":
                for layer in range(layers):
                    # random e4m3 bytes with the exponent capped (no NaN / huge values) and scales near 1 / 448
                    self.kv8.data[layer].random_(0, 256).bitwise_and_(0xBF)
                    self.kv8.scales[layer].uniform_(0.004, 0.012)
        else:
            pool_shape = (layers, self.total_pages, self.local_kv_heads, shape.page, shape.head_dim)
            self.key_blocks = torch.empty(pool_shape, dtype=torch.bfloat16, device=self.device)
            self.value_blocks = torch.empty(pool_shape, dtype=torch.bfloat16, device=self.device)
            if kv_init == "zeros":
                self.key_blocks.zero_()
                self.value_blocks.zero_()
            elif kv_init == "normal":
                for pool in (self.key_blocks, self.value_blocks):
                    for layer in range(layers):
                        pool[layer].normal_()
        self.rope = rope_table(shape, max_context, self.device)
        self.scratch = decode_scratch(max(max_batch, self.decode_buckets[-1]), self.local_q_heads,
                                      self.local_kv_heads, shape.head_dim, max_batch * max_context, self.device)
        # lm_head + greedy sampling: one pass over the tied embedding that never writes the logits
        # (mie_lm_head_argmax) unless MIE_LM_HEAD=cublas.
        self.fused_lm_head = os.environ.get("MIE_LM_HEAD", "fused") != "cublas"
        # Tensor parallel decode: the all-reduce after o_proj / down_proj is fused into the residual add +
        # RMSNorm + quantisation kernel over peer memory unless MIE_TP_EXCHANGE=nccl (or fused_exchange=False).
        if fused_exchange is None:
            fused_exchange = os.environ.get("MIE_TP_EXCHANGE", "fused") != "nccl"
        self.exchange = None
        if self.tp > 1 and fused_exchange:
            # Rows for the largest decode bucket plus the largest prompt-chunk bucket of a mixed step; a longer
            # flat forward (a whole-prompt prefill) sums its partial rows with NCCL instead.
            exchange_rows = max(max_batch, self.decode_buckets[-1]) + max(self.chunk_buckets, default=0)
            self.exchange = PeerExchange(self.tp, weights.tp_rank, exchange_rows, shape.hidden, self.device,
                                         process_group)

    # -- small helpers ------------------------------------------------------------------------

    def _quant_buffers(self, rows: int, width: int) -> tuple[torch.Tensor, torch.Tensor]:
        padded = (width + 15) // 16 * 16
        q = torch.empty(rows, padded, dtype=torch.float8_e4m3fn, device=self.device)
        if padded != width:
            q.view(torch.uint8)[:, width:].zero_()
        return q, torch.empty((width + 127) // 128, rows, dtype=torch.float32, device=self.device)

    def _norm(self, x, weight, residual=None, *, quantize: bool):
        """(normed bf16 or None, summed or None, quantised pair or None)."""

        rows, cols = x.shape
        lib, stream = _lib.load(), _lib.stream_arg(self.device)
        summed = torch.empty_like(x) if residual is not None else None
        if quantize:
            q, scales = self._quant_buffers(rows, cols)
            _lib.check(lib.mie_rms_norm(_lib.ptr(x), x.stride(0), _lib.ptr(residual), _lib.ptr(summed),
                                        _lib.ptr(weight), None, _lib.ptr(q), q.stride(0), _lib.ptr(scales),
                                        scales.stride(0), rows, cols, self.shape.rms_eps, stream))
            return None, summed, (q, scales)
        out = torch.empty_like(x)
        _lib.check(lib.mie_rms_norm(_lib.ptr(x), x.stride(0), _lib.ptr(residual), _lib.ptr(summed),
                                    _lib.ptr(weight), _lib.ptr(out), None, 0, None, 0, rows, cols,
                                    self.shape.rms_eps, stream))
        return out, summed, None

    def _gemm(self, quantized, weight, weight_scale, rows: int, k: int, out: torch.Tensor | None = None) -> torch.Tensor:
        if out is None:
            out = torch.empty(rows, weight.shape[0], dtype=torch.bfloat16, device=self.device)
        sm89_fp8.launch_fp8_gemm(quantized[0], quantized[1], weight, weight_scale, out, rows, k, status=self.status)
        return out

    def _quantize(self, x: torch.Tensor):
        return sm89_fp8.quantize_activation_kmajor(x)

    def _all_reduce(self, x: torch.Tensor) -> torch.Tensor:
        if self.tp > 1:
            torch.distributed.all_reduce(x, group=self.group)
        return x

    def _silu_mul_quantized(self, gate_up: torch.Tensor, rows: int):
        """SiLU(gate) * up over the two windows of the merged gate_up output, quantised for down_proj."""

        inter = self.local_inter
        q, scales = self._quant_buffers(rows, inter)
        _lib.check(_lib.load().mie_silu_mul(_lib.ptr(gate_up), _lib.ptr(gate_up[:, inter:]), gate_up.stride(0), None,
                                            _lib.ptr(q), q.stride(0), _lib.ptr(scales), scales.stride(0), rows,
                                            inter, _lib.stream_arg(self.device)))
        return q, scales

    def _row_parallel_then_norm(self, quantized, weight, weight_scale, rows: int, k: int, residual, norm_weight,
                                *, quantize: bool):
        """Row-parallel projection, sum over the ranks, residual add and RMSNorm of the sum.  Returns
        ``(normed bf16 or None, new residual, quantised pair or None)`` like ``_norm``.  With the fused exchange
        the new residual is only valid in the rows this rank owns (the only rows it reads again)."""

        ex = self.exchange
        if ex is None or rows > ex.max_rows:
            out = self._all_reduce(self._gemm(quantized, weight, weight_scale, rows, k))
            return self._norm(out, norm_weight, residual, quantize=quantize)
        self._gemm(quantized, weight, weight_scale, rows, k, out=ex.partial[:rows])
        summed = torch.empty_like(residual)
        ex.reduce_norm(rows, residual, summed, norm_weight, self.shape.rms_eps, quantized=quantize, status=self.status)
        if quantize:
            return None, summed, (ex.q[:rows], ex.scales[:, :rows])
        return ex.normed[:rows], summed, None

    def _qkv_post(self, layer_index: int, layer, qkv, queries, positions, token_to_sequence, block_tables,
                  tokens: int, table_rows: int) -> None:
        """q/k RMSNorm + RoPE on the merged qkv rows, K/V rows to their page slots, q rows to ``queries``."""

        shape = self.shape
        if self.kv8 is not None:
            _lib.check(_lib.load().mie_qkv_norm_rope_write_kv8(
                _lib.ptr(qkv), qkv.stride(0), _lib.ptr(layer.q_norm), _lib.ptr(layer.k_norm), _lib.ptr(self.rope),
                int(self.rope.shape[0]), _lib.index_arg(positions), _lib.index_arg(token_to_sequence),
                _lib.index_arg(block_tables), _lib.ptr(queries), _lib.ptr(self.kv8.data[layer_index]),
                self.kv8.page_stride_bytes, _lib.ptr(self.kv8.scales[layer_index]), tokens, self.local_q_heads,
                self.local_kv_heads, self.total_pages, table_rows, int(block_tables.shape[1]), shape.rms_eps,
                _lib.ptr(self.status), _lib.stream_arg(self.device)))
            return
        _lib.check(_lib.load().mie_qkv_norm_rope_write(
            _lib.ptr(qkv), qkv.stride(0), _lib.ptr(layer.q_norm), _lib.ptr(layer.k_norm), _lib.ptr(self.rope),
            int(self.rope.shape[0]), _lib.index_arg(positions), _lib.index_arg(token_to_sequence),
            _lib.index_arg(block_tables), _lib.ptr(queries), _lib.view4_arg(self.key_blocks[layer_index]),
            _lib.view4_arg(self.value_blocks[layer_index]), tokens, self.local_q_heads, self.local_kv_heads,
            shape.page, self.total_pages, table_rows, int(block_tables.shape[1]), shape.rms_eps,
            _lib.ptr(self.status), _lib.stream_arg(self.device)))

    # -- the decode forward -------------------------------------------------------------------

    def decode_forward(self, input_ids: torch.Tensor, sequence_lengths: torch.Tensor,
                       block_tables: torch.Tensor, return_logits: bool = False):
        """One token per request.  ``sequence_lengths`` already counts the new token, which is
        written at position ``length - 1``.  Returns the greedy next token ids ``[batch]`` (int64)."""

        shape, lib = self.shape, _lib.load()
        batch = int(input_ids.shape[0])
        launches_before = lib.mie_launch_count()
        hd, lq = shape.head_dim, self.local_q_heads
        hidden = self.weights.embedding.index_select(0, input_ids)
        positions = sequence_lengths - 1
        scale = 1.0 / math.sqrt(hd)
        layers = self.weights.layers
        _, _, quantized = self._norm(hidden, layers[0].input_norm, quantize=True)
        residual, final = hidden, None
        for index, layer in enumerate(layers):
            qkv = self._gemm(quantized, layer.qkv, layer.qkv_scale, batch, shape.hidden)
            queries = torch.empty(batch, lq, 1, hd, dtype=torch.bfloat16, device=self.device)
            self._qkv_post(index, layer, qkv, queries, positions, None, block_tables, batch, batch)
            attended = torch.empty_like(queries)
            attn_q = self._quant_buffers(batch, lq * hd)
            if self.kv8 is not None:
                launch_decode_attention_kv8(queries, attended, self.kv8.data[index], self.kv8.scales[index],
                                            block_tables, sequence_lengths, None, scale=scale, scratch=self.scratch,
                                            split_policy=1, use_plan=index % PLAN_SLOTS != 0,
                                            plan_slot=index % PLAN_SLOTS, status=self.status, quantized_out=attn_q)
            else:
                launch_decode_attention(queries, attended, self.key_blocks[index], self.value_blocks[index],
                                        block_tables, sequence_lengths, None, scale=scale,
                                        max_total_tokens=batch * self.max_context, scratch=self.scratch,
                                        split_policy=1, use_plan=index % PLAN_SLOTS != 0,
                                        plan_slot=index % PLAN_SLOTS, status=self.status,
                                        quantized_out=attn_q)
            _, residual, quantized = self._row_parallel_then_norm(attn_q, layer.o, layer.o_scale, batch, lq * hd,
                                                                  residual, layer.post_norm, quantize=True)
            gate_up = self._gemm(quantized, layer.gate_up, layer.gate_up_scale, batch, shape.hidden)
            act_q = self._silu_mul_quantized(gate_up, batch)
            last = index + 1 == len(layers)
            next_norm = self.weights.final_norm if last else layers[index + 1].input_norm
            final, residual, quantized = self._row_parallel_then_norm(act_q, layer.down, layer.down_scale, batch,
                                                                      self.local_inter, residual, next_norm,
                                                                      quantize=not last)
        if self.fused_lm_head and not return_logits and batch <= 256:
            tokens = self.greedy_tokens(final)
            self.launches_per_step = int(lib.mie_launch_count() - launches_before)
            return tokens
        logits = torch.matmul(final, self.weights.lm_head.t())
        self.launches_per_step = int(lib.mie_launch_count() - launches_before)
        if self.tp == 1:
            tokens = logits.argmax(dim=-1)
            return (tokens, logits) if return_logits else tokens
        return sharded_greedy_tokens(logits, self.weights.vocab_start, self.tp, self.group)

    def greedy_tokens(self, final: torch.Tensor) -> torch.Tensor:
        """Greedy next tokens of normed hidden rows ``[rows, hidden]`` (rows <= 256): the bf16 product with the
        tied lm_head and its argmax in one pass (reference: engine/model_runner/qwen3_mixed.py:164-174)."""

        values = torch.empty(final.shape[0], dtype=torch.int32, device=self.device) if self.tp > 1 else None
        tokens = self.lm_head_argmax(final, self.weights.lm_head, self.weights.vocab_start, values)
        return sharded_greedy_from_pairs(tokens, values, self.tp, self.group) if self.tp > 1 else tokens

    # -- flat forward: decode rows and packed prompt chunks in one token stream --------------------------

    def mixed_forward(self, input_ids: torch.Tensor, token_to_sequence: torch.Tensor,
                      token_positions: torch.Tensor, block_tables: torch.Tensor, *, decode_rows: int,
                      decode_lengths: torch.Tensor | None, cu_seqlens: torch.Tensor, kv_lens: torch.Tensor,
                      max_query_len: int, logit_rows: torch.Tensor, return_logits: bool = False):
        """One flat ``[tokens]`` forward (reference: engine/model_runner/qwen3_mixed.py:125-178 and the mixed
        branch of the attention adapter, engine/kv_cache/qwen3_paged.py:221-330).

        Tokens ``[0, decode_rows)`` are decode tokens, one per request: token ``i`` belongs to table row ``i``
        and sits at position ``decode_lengths[i] - 1``.  The remaining tokens are prompt chunks packed back to
        back; ``cu_seqlens`` (relative to the first chunk token) and ``kv_lens`` describe them, their table rows
        follow the decode rows, ``token_to_sequence`` / ``token_positions`` place every token's K/V.  Per layer
        the K/V rows of ALL tokens are scattered first, then the decode rows run the paged decode kernel and
        the chunk rows the tiled prefill kernel (causal within the chunk, over the request's cached prefix);
        all other operators run once over the whole stream.  ``logit_rows`` selects the rows that are
        projected to logits; their greedy tokens are returned in that order."""

        shape, lib = self.shape, _lib.load()
        stream = _lib.stream_arg(self.device)
        tokens = int(input_ids.shape[0])
        table_rows = int(block_tables.shape[0])
        chunk_tokens = tokens - decode_rows
        hd, lq = shape.head_dim, self.local_q_heads
        launches_before = lib.mie_launch_count()
        hidden = self.weights.embedding.index_select(0, input_ids)
        scale = 1.0 / math.sqrt(hd)
        layers = self.weights.layers
        # Same layer structure as the decode forward: every residual add + RMSNorm (+ quantisation) is fused
        # with the sum over the ranks that precedes it (the peer-memory exchange when the token count fits its
        # buffers, NCCL all-reduce + the norm kernel otherwise).
        _, _, quantized = self._norm(hidden, layers[0].input_norm, quantize=True)
        residual, normed = hidden, None
        chunk_tables = block_tables[decode_rows:]
        if self.kv8 is not None and chunk_tokens:
            # The chunk kernel reads bf16 pages: per layer, after the writer has quantised the new rows into the
            # FP8 pool, the chunk requests' pages (cached prefix and the chunk itself) are dequantised into a
            # staging set of bf16 pages addressed by a renumbered table, so a chunk attends exactly what the
            # cache holds, as the decode steps after it will.
            staged_ids = chunk_tables.clamp_min(0).flatten().long()
            numbering = torch.arange(staged_ids.numel(), dtype=chunk_tables.dtype, device=self.device)
            chunk_tables = torch.where(chunk_tables >= 0, numbering.view_as(chunk_tables),
                                       torch.full_like(chunk_tables, -1))
        for index, layer in enumerate(layers):
            qkv = self._gemm(quantized, layer.qkv, layer.qkv_scale, tokens, shape.hidden)
            queries = torch.empty(tokens, lq, hd, dtype=torch.bfloat16, device=self.device)
            self._qkv_post(index, layer, qkv, queries, token_positions, token_to_sequence, block_tables, tokens,
                           table_rows)
            attended = torch.empty_like(queries)
            if decode_rows and self.kv8 is not None:
                launch_decode_attention_kv8(queries[:decode_rows].unsqueeze(2), attended[:decode_rows].unsqueeze(2),
                                            self.kv8.data[index], self.kv8.scales[index], block_tables[:decode_rows],
                                            decode_lengths, None, scale=scale, scratch=self.scratch, split_policy=1,
                                            use_plan=index % PLAN_SLOTS != 0, plan_slot=index % PLAN_SLOTS,
                                            status=self.status)
            elif decode_rows:
                launch_decode_attention(queries[:decode_rows].unsqueeze(2), attended[:decode_rows].unsqueeze(2),
                                        self.key_blocks[index], self.value_blocks[index],
                                        block_tables[:decode_rows], decode_lengths, None, scale=scale,
                                        max_total_tokens=decode_rows * self.max_context, scratch=self.scratch,
                                        split_policy=1, use_plan=index % PLAN_SLOTS != 0,
                                        plan_slot=index % PLAN_SLOTS, status=self.status)
            if chunk_tokens:
                if self.kv8 is not None:
                    key_pages, value_pages = self.kv8.dequantized_pages(index, staged_ids)
                else:
                    key_pages, value_pages = self.key_blocks[index], self.value_blocks[index]
                launch_flash_prefill(queries[decode_rows:], attended[decode_rows:], key_pages, value_pages,
                                     chunk_tables, cu_seqlens, kv_lens, max_query_len=max_query_len, scale=scale,
                                     status=self.status)
            attn_q = self._quantize(attended.view(tokens, lq * hd))
            _, residual, quantized = self._row_parallel_then_norm(attn_q, layer.o, layer.o_scale, tokens, lq * hd,
                                                                  residual, layer.post_norm, quantize=True)
            gate_up = self._gemm(quantized, layer.gate_up, layer.gate_up_scale, tokens, shape.hidden)
            act_q = self._silu_mul_quantized(gate_up, tokens)
            last = index + 1 == len(layers)
            next_norm = self.weights.final_norm if last else layers[index + 1].input_norm
            normed, residual, quantized = self._row_parallel_then_norm(act_q, layer.down, layer.down_scale, tokens,
                                                                       self.local_inter, residual, next_norm,
                                                                       quantize=not last)
        final = normed.index_select(0, logit_rows)
        if self.fused_lm_head and not return_logits and final.shape[0] <= 256:
            picked = self.greedy_tokens(final)
            self.launches_per_step = int(lib.mie_launch_count() - launches_before)
            return picked
        logits = torch.matmul(final, self.weights.lm_head.t())
        self.launches_per_step = int(lib.mie_launch_count() - launches_before)
        picked = sharded_greedy_tokens(logits, self.weights.vocab_start, self.tp, self.group)
        return (picked, logits) if return_logits else picked


__all__ = ["DEFAULT_DECODE_BUCKETS", "DecodeBuffers", "LayerWeights", "MixedBuffers", "PADDING", "Qwen3DecodeRunner",
           "Qwen3Shape", "Qwen3Weights", "scale_window", "select_bucket", "shard_bounds",
           "quantize_weight_blocks", "rope_table", "sharded_greedy_from_pairs", "sharded_greedy_tokens"]

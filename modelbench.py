"""Prefill and decode throughput of a model design at layer sizes of real models, beside the framework's closest other
design at equal sizes, and every kernel of both against its roofline: Tidelorn beside the Qwen3 runner
(``bench.py --workload tidelorn``), Ripesun beside Tidelorn (``--workload ripesun``).

Random weights.  ``Tidelorn`` here alternates whole-prefix and 1,024-token-window layers (beside Ripesun, whose
attention layers all have such a window, windowed layers only).  Decode is a replayed CUDA
graph of one step at a uniform context; prefill is one packed forward of whole prompts.  Kernels are timed alone with
CUDA events, L2 flushed before each (median of the repeats): a kernel's fraction is (bytes / time / copy peak) or
(FLOPs / time / tensor peak).
"""

from __future__ import annotations

import gc
import statistics

import torch

from mini_inference_engine_b200.engine.kernels.decoder_glue import (
    clamped_glu,
    embed_tokens,
    gated_rms_norm,
    gelu,
    qkv_norm_mix_write,
    residual_norm_,
    sum_rms_norm,
)
from mini_inference_engine_b200.engine.kernels.recurrence import gated_average, outer_recurrence
from mini_inference_engine_b200.engine.kv_cache.latent_attention import (
    VisibleSpans,
    latent_decode_attention,
    latent_decode_scratch,
    latent_norm_write,
    rotate_heads,
)
from mini_inference_engine_b200.engine.kv_cache.sink_attention import sink_decode_attention, sink_prefill_attention
from mini_inference_engine_b200.engine.kv_cache.triton_flash_prefill import launch_flash_prefill
from mini_inference_engine_b200.engine.kv_cache.triton_paged_attention import decode_scratch, launch_decode_attention
from mini_inference_engine_b200.engine.model_runner.qwen3_decode import Qwen3DecodeRunner, Qwen3Shape, Qwen3Weights
from mini_inference_engine_b200.engine.model_runner.ripesun import RipesunRunner, RipesunShape, RipesunWeights
from mini_inference_engine_b200.engine.model_runner.tidelorn import TidelornRunner, TidelornShape, TidelornWeights

# name: width, query heads, key/value heads, head size, feed-forward, vocabulary
SIZES = {
    "1.7b-layers": (2048, 16, 8, 128, 6144, 151936),
    "4b-layers": (2560, 32, 8, 128, 9728, 151936),
    "8b-layers": (4096, 32, 8, 128, 12288, 151936),
}
LAYERS = 8
WINDOW = 1024


def tidelorn_config(width, heads, kv_heads, dim, ff, vocab, layers=LAYERS, window=WINDOW, windowed_only=False) -> dict:
    entries = []
    for index in range(layers):
        mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "v_mix": True}
        if index % 2 == 0 and not windowed_only:
            mixer["q_temp"] = {"coef": 0.1, "every": 4096}
        else:
            mixer["mask"] = {"size": window}
        entries.append({"type": "attention" if "q_temp" in mixer else "attention_2", "mixer": mixer,
                        "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}})
    return {"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "postln_alpha": 2.0, "layers": entries,
            "embedding": {"scale": width ** 0.5, "bigram": {"buckets": 65521, "mul_prev": 8191, "mul_cur": 127}}}


def _tables(batch: int, pages_each: int, total: int, device) -> torch.Tensor:
    order = torch.randperm(total, generator=torch.Generator().manual_seed(1))[:batch * pages_each]
    return order.to(torch.int32).view(batch, pages_each).to(device)


def _event_ms(run, repeats: int, device) -> float:
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    for _ in range(repeats):
        run()
    end.record()
    torch.cuda.synchronize(device)
    return start.elapsed_time(end) / repeats


class Flusher:
    """Between two launches a buffer of twice the L2 is read, so that nothing of the kernel's data is left in L2 and no
    dirty lines are either (a kernel that reads less than the L2 holds would pay for writing them back)."""

    def __init__(self, device) -> None:
        self.device, self.buffer = device, torch.zeros(64 << 20, dtype=torch.int32, device=device)

    def median_us(self, run, repeats: int = 9) -> float:
        for _ in range(3):
            run()
        samples = []
        for _ in range(repeats):
            self.buffer.max()
            samples.append(_event_ms(run, 1, self.device) * 1e3)
        return statistics.median(samples)


def _throughput(runner, vocab: int, batch: int, context: int, prompts: int, prompt_len: int, steps: int, device) -> dict:
    page = runner.shape.page
    pages_each = -(-(context + steps + 16) // page)
    buffers = runner.capture(batch, pages_each, advance=True)
    launches = runner.launches_per_step
    buffers.block_tables.copy_(_tables(batch, pages_each, runner.num_pages, device))
    buffers.input_ids.copy_(torch.randint(0, vocab, (batch,), device=device))
    buffers.sequence_lengths.fill_(context + 1)
    extra = {}
    if runner.recurrent:
        buffers.state_slots.copy_(torch.arange(batch, dtype=torch.int32))
        extra["state_slots"] = torch.arange(prompts, dtype=torch.int32, device=device)
    if runner.wants_chunk_starts:
        extra["chunk_starts"] = [0] * prompts
    for _ in range(3):
        runner.replay(batch, advance=True)
    torch.cuda.synchronize(device)
    decode_ms = _event_ms(lambda: runner.replay(batch, advance=True), steps, device)
    tokens = prompts * prompt_len
    ids = torch.randint(0, vocab, (tokens,), device=device)
    owners = torch.arange(prompts, dtype=torch.int32, device=device).repeat_interleave(prompt_len)
    positions = torch.arange(prompt_len, dtype=torch.int32, device=device).repeat(prompts)
    tables = _tables(prompts, -(-prompt_len // page), runner.num_pages, device)
    cu = torch.arange(prompts + 1, dtype=torch.int32, device=device) * prompt_len
    lens = torch.full((prompts,), prompt_len, dtype=torch.int32, device=device)

    def prefill():
        runner.prefill_forward(ids, owners, positions, tables, cu, lens, prompt_len, **extra)

    for _ in range(3):
        prefill()
    torch.cuda.synchronize(device)
    prefill_ms = _event_ms(prefill, 5, device)
    runner.check_status()
    return {"decode": {"ms_per_step": decode_ms, "tok_per_s": batch / decode_ms * 1e3,
                       "launches_of_this_library": launches},
            "prefill": {"ms": prefill_ms, "tok_per_s": tokens / prefill_ms * 1e3}}


def _row(us: float, *, bytes_: float = 0.0, flops: float = 0.0, hbm: float, tensor: float) -> dict:
    """Time beside the roofline time max(bytes / copy peak, FLOPs / tensor peak) of the same work."""

    floor = max(bytes_ / (hbm * 1e9), flops / (tensor * 1e12)) * 1e6
    return {"us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3)}


def _kernels(size, tide: TidelornRunner, qwen: Qwen3DecodeRunner, batch, context, prompts, prompt_len, hbm, tensor,
             device) -> dict:
    width, heads, kv, dim, ff, vocab = size
    flush, page = Flusher(device), tide.shape.page
    w, q = tide.weights.layers[0], qwen.weights.layers[0]
    layer = tide.shape.layers[0]
    out = {}

    def pair(name, ours, theirs, *, work, their_work=None):
        their_work = their_work or work
        a = _row(flush.median_us(ours), hbm=hbm, tensor=tensor, **work)
        b = _row(flush.median_us(theirs), hbm=hbm, tensor=their_work.pop("tensor", tensor), **their_work)
        out[name] = {"tidelorn": a, "qwen3": b, "distance_ratio": round(b["frac"] / a["frac"], 2)}

    def bf16(*shape):
        return torch.randn(*shape, device=device).to(torch.bfloat16)

    # Decode attention over a uniform context, and the windowed form of it.
    tables = _tables(batch, -(-context // page), tide.num_pages, device)
    lengths = torch.full((batch,), context, dtype=torch.int32, device=device)
    queries, attended = bf16(batch, heads, dim), bf16(batch, heads, dim)
    kv_bytes = 2 * kv * dim * 2

    def tide_decode(window):
        key = next(k for k, layer in zip((a[0] for a in tide._attention), tide.shape.layers) if layer.window == window)
        return lambda: sink_decode_attention(queries, attended, tide.key_blocks[0], tide.value_blocks[0], tables,
                                             lengths, scale=layer.scale, window=window, sinks=w.sinks,
                                             scratch=tide._scratch[key], status=tide.status)

    def qwen_decode():
        launch_decode_attention(queries.unsqueeze(2), attended.unsqueeze(2), qwen.key_blocks[0], qwen.value_blocks[0],
                                tables, lengths, None, scale=layer.scale, max_total_tokens=batch * context,
                                scratch=qwen.scratch, split_policy=1, status=qwen.status)

    pair("decode attention", tide_decode(None), qwen_decode, work={"bytes_": batch * context * kv_bytes})
    reach = min(context, WINDOW)
    pair("decode attention, window", tide_decode(WINDOW), qwen_decode, work={"bytes_": batch * reach * kv_bytes},
         their_work={"bytes_": batch * context * kv_bytes})

    # Prefill attention of whole prompts.
    tokens = prompts * prompt_len
    queries_p, attended_p = bf16(tokens, heads, dim), bf16(tokens, heads, dim)
    tables_p = _tables(prompts, -(-prompt_len // page), tide.num_pages, device)
    cu = torch.arange(prompts + 1, dtype=torch.int32, device=device) * prompt_len
    lens = torch.full((prompts,), prompt_len, dtype=torch.int32, device=device)

    def tide_prefill(window):
        return lambda: sink_prefill_attention(queries_p, attended_p, tide.key_blocks[0], tide.value_blocks[0], tables_p,
                                              cu, lens, max_query_len=prompt_len, scale=layer.scale, window=window,
                                              sinks=w.sinks, status=tide.status)

    def qwen_prefill():
        launch_flash_prefill(queries_p, attended_p, qwen.key_blocks[0], qwen.value_blocks[0], tables_p, cu, lens,
                             max_query_len=prompt_len, scale=layer.scale, status=qwen.status)

    seen = prompts * prompt_len * (prompt_len + 1) / 2
    inside = prompts * (WINDOW * prompt_len - WINDOW * (WINDOW - 1) / 2 if prompt_len > WINDOW
                        else prompt_len * (prompt_len + 1) / 2)
    pair("prefill attention", tide_prefill(None), qwen_prefill, work={"flops": 4 * heads * dim * seen})
    pair("prefill attention, window", tide_prefill(WINDOW), qwen_prefill, work={"flops": 4 * heads * dim * inside},
         their_work={"flops": 4 * heads * dim * seen})

    # Projections: bf16 library products against the FP8 kernel (its peak taken as twice the bf16 one).
    for rows, label in ((batch, "decode"), (tokens, "prefill")):
        for name, weight, bias, q8, q8s in (("qkv", w.qkv, w.qkv_bias, q.qkv, q.qkv_scale), ("o", w.o, None, q.o, q.o_scale),
                                            ("gate_up", w.gate_up, None, q.gate_up, q.gate_up_scale),
                                            ("down", w.down, None, q.down, q.down_scale)):
            n, k = weight.shape
            x = bf16(rows, k)
            x8 = qwen._quantize(x)
            pair(f"{label} {name} projection", lambda: tide._linear(x, weight, bias),
                 lambda: qwen._gemm(x8, q8, q8s, rows, k),
                 work={"bytes_": 2 * (n * k + rows * (n + k)), "flops": 2 * rows * n * k},
                 their_work={"bytes_": n * k + rows * (2 * n + k), "flops": 2 * rows * n * k, "tensor": 2 * tensor})
        qkv = bf16(rows, w.qkv.shape[0])
        pos = (lengths - 1) if label == "decode" else torch.arange(prompt_len, dtype=torch.int32, device=device).repeat(prompts)
        own = None if label == "decode" else torch.arange(prompts, dtype=torch.int32, device=device).repeat_interleave(prompt_len)
        tab, q_out = (tables, queries) if label == "decode" else (tables_p, queries_p)
        pair(f"{label} q/k norm, mix, page write",
             lambda: qkv_norm_mix_write(qkv, q_out, tide.key_blocks[0], tide.value_blocks[0], pos, own, tab, q_heads=heads,
                                        kv_heads=kv, dim=dim, value_dim=dim, unit_norm=True, eps=1e-6,
                                        temperature=layer.temperature, v_first=qkv[:, (heads + kv) * dim:], lam=0.5,
                                        status=tide.status),
             lambda: qwen._qkv_post(0, q, qkv, q_out, pos, own, tab, rows, tab.shape[0]),
             work={"bytes_": 4 * rows * w.qkv.shape[0]})
        x32, y = torch.randn(rows, width, device=device), bf16(rows, width)
        xb = x32.to(torch.bfloat16)
        pair(f"{label} residual sum + norm", lambda: sum_rms_norm(x32, y, w.norm1, eps=1e-6, alpha=2.0, weight_offset=1.0),
             lambda: qwen._norm(xb, q.input_norm, y, quantize=True), work={"bytes_": rows * width * 12},
             their_work={"bytes_": rows * width * 7})
        gate_up = bf16(rows, 2 * ff)
        pair(f"{label} gate", lambda: clamped_glu(gate_up, limit=7.0, slope=1.702, up_offset=1.0),
             lambda: qwen._silu_mul_quantized(gate_up, rows), work={"bytes_": rows * ff * 6},
             their_work={"bytes_": rows * ff * 5})
        ids = torch.randint(0, vocab, (rows,), device=device)
        pair(f"{label} embedding",
             lambda: embed_tokens(ids, tide.weights.embed, pos, own, tab, scale=2.0, page=page, num_pages=tide.total_pages,
                                  bigram=tide.weights.bigram, mul_prev=8191, mul_cur=127, history=tide.history,
                                  turns=tide.weights.turns, status=tide.status),
             lambda: qwen.weights.embedding.index_select(0, ids), work={"bytes_": rows * width * 10},
             their_work={"bytes_": rows * width * 4})
        del qkv, x32, y, xb, gate_up
    final = bf16(batch, width)
    pair("lm_head + greedy", lambda: tide.lm_head_argmax(final, tide.weights.head), lambda: qwen.greedy_tokens(final),
         work={"bytes_": 2 * vocab * width})
    tide.check_status()
    qwen.check_status()
    return out


# Head sizes that are not two 64-dim boxes: key size, value size.
HEAD_SIZES = ((64, 64), (96, 96), (192, 128), (256, 256))


def head_sizes(device, hbm: float, tensor: float, *, heads: int = 32, kv: int = 8, batch: int = 64, context: int = 2048,
               prompts: int = 4, prompt_len: int = 2048) -> dict:
    """The two streaming attention kernels at other head sizes (whole prefix)."""

    flush, out = Flusher(device), {}
    pages = batch * (context // 16) + 8
    tables = _tables(batch, context // 16, pages, device)
    lengths = torch.full((batch,), context, dtype=torch.int32, device=device)
    cu = torch.arange(prompts + 1, dtype=torch.int32, device=device) * prompt_len
    status = torch.zeros(1, dtype=torch.int32, device=device)
    sinks = torch.zeros(heads, device=device)
    for dim, vdim in HEAD_SIZES:
        keys, values = (torch.randn(pages, kv, 16, n, device=device).to(torch.bfloat16) for n in (dim, vdim))
        scratch = decode_scratch(batch, heads, kv, vdim, batch * context, device)
        common = dict(scale=dim ** -0.5, sinks=sinks, status=status)
        rows = prompts * prompt_len
        query, result = (torch.randn(rows, heads, n, device=device).to(torch.bfloat16) for n in (dim, vdim))
        decode = flush.median_us(lambda: sink_decode_attention(query[:batch], result[:batch], keys, values, tables,
                                                               lengths, scratch=scratch, **common))
        prefill = flush.median_us(lambda: sink_prefill_attention(query, result, keys, values, tables[:prompts], cu,
                                                                 lengths[:prompts], max_query_len=prompt_len, **common))
        flops = 2 * heads * (dim + vdim) * prompts * prompt_len * (prompt_len + 1) / 2
        out[f"{dim}/{vdim}"] = {
            "decode": _row(decode, bytes_=batch * context * kv * (dim + vdim) * 2, hbm=hbm, tensor=tensor),
            "prefill": _row(prefill, flops=flops, hbm=hbm, tensor=tensor)}
    return out


def run(device, hbm: float, tensor: float, *, sizes=tuple(SIZES), batch: int = 64, context: int = 2048, prompts: int = 8,
        prompt_len: int = 2048, steps: int = 50) -> dict:
    result = {"layers": LAYERS, "window": WINDOW, "decode_batch": batch, "decode_context": context,
              "prefill": f"{prompts} x {prompt_len}", "hbm_gb_s": hbm, "bf16_tflop_s": tensor, "sizes": {},
              "head_sizes": head_sizes(device, hbm, tensor)}
    for name in sizes:
        width, heads, kv, dim, ff, vocab = size = SIZES[name]
        pages = max(batch * (-(-(context + steps + 16) // 16)), prompts * (-(-prompt_len // 16))) + 8
        options = dict(num_pages=pages, max_batch=batch, max_context=context + steps + 64)
        shape = TidelornShape.from_config(tidelorn_config(*size))
        tide = TidelornRunner(TidelornWeights.random(shape, device), kv_init="normal", **options)
        entry = {"tidelorn": _throughput(tide, vocab, batch, context, prompts, prompt_len, steps, device)}
        tide.release_graphs()
        q_shape = Qwen3Shape(layers=LAYERS, hidden=width, q_heads=heads, kv_heads=kv, head_dim=dim, intermediate=ff,
                             vocab=vocab)
        qwen = Qwen3DecodeRunner(Qwen3Weights(q_shape, device), kv_init="normal", **options)
        entry["qwen3_fp8"] = _throughput(qwen, vocab, batch, context, prompts, prompt_len, steps, device)
        qwen.release_graphs()
        entry["kernels"] = _kernels(size, tide, qwen, batch, context, prompts, prompt_len, hbm, tensor, device)
        result["sizes"][name] = entry
        del tide, qwen
        gc.collect()
        torch.cuda.empty_cache()
    return result


# Ripesun beside Tidelorn.  name: width, heads, feed-forward, query latent, vocabulary; heads of 128 + 64 rotated query /
# key and 128 value entries over a 512-entry latent, recurrent heads of 128 x 128, channels as wide as the stream.
RIPESUN_SIZES = {
    "2048-wide": (2048, 16, 6144, 768, 151936),
    "4096-wide": (4096, 32, 12288, 1536, 151936),
}
HEAD, ROTATED, KV_RANK, SIDE = 128, 64, 512, 256


def ripesun_config(width, heads, ff, q_rank, vocab, window=WINDOW) -> dict:
    """Eight layers: latent attention, two outer recurrences, a gated average, and the same again with the second
    attention layer reading the first one's rows."""

    mlp = {"kind": "dense", "ff": ff}
    latent = {"heads": heads, "dim": HEAD, "rot_dim": ROTATED, "vdim": HEAD, "q_rank": q_rank, "kv_rank": KV_RANK,
              "scale": (HEAD + ROTATED) ** -0.5, "mask": {"size": window}, "rot": {"base": 1e6, "dims": ROTATED}}
    outer = {"heads": heads, "dim": HEAD, "vdim": HEAD, "decay": [1.0 - 2.0 ** -(5 + i % 8) for i in range(heads)]}
    recurrent = [{"type": "lightning", "mixer": outer, "mlp": mlp}] * 2 + [
        {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}]
    entries = [{"type": "latent_attention", "mixer": latent, "mlp": mlp}, *recurrent,
               {"type": "latent_attention", "mixer": {**latent, "kv_from": 0}, "mlp": mlp}, *recurrent]
    return {"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "layers": entries,
            "embedding": {"scale": width ** 0.5}, "token_side": {"dim": SIDE}, "logit_softcap": 30.0}


def _ripesun_kernels(size, ripe: RipesunRunner, tide: TidelornRunner, batch, context, prompts, prompt_len, hbm, tensor,
                     device) -> dict:
    """Every kernel of Ripesun with its roofline, and beside it the kernel of Tidelorn that does the like work."""

    width, heads, ff, q_rank, vocab = size
    flush, page, out, window = Flusher(device), ripe.shape.page, {}, WINDOW
    w, outer, average = ripe.weights.layers[0], ripe.weights.layers[1], ripe.weights.layers[3]
    t = tide.weights.layers[0]
    mixer, values = ripe.shape.layers[0].mixer, heads * HEAD

    def pair(name, ours, theirs, *, work, their_work=None):
        a = _row(flush.median_us(ours), hbm=hbm, tensor=tensor, **work)
        b = _row(flush.median_us(theirs), hbm=hbm, tensor=tensor, **(their_work or work))
        out[name] = {"ripesun": a, "tidelorn": b, "distance_ratio": round(b["frac"] / a["frac"], 2)}

    def bf16(*shape):
        return torch.randn(*shape, device=device).to(torch.bfloat16)

    kv = tide.shape.layers[0].kv_heads
    t_heads, t_dim = tide.shape.layers[0].heads, tide.shape.layers[0].dim
    reach = min(context, window)
    tokens = prompts * prompt_len
    inside = prompts * (window * prompt_len - window * (window - 1) / 2 if prompt_len > window
                        else prompt_len * (prompt_len + 1) / 2)
    tables = _tables(batch, -(-context // page), ripe.num_pages, device)
    lengths = torch.full((batch,), context, dtype=torch.int32, device=device)
    tables_p = _tables(prompts, -(-prompt_len // page), ripe.num_pages, device)
    cu = torch.arange(prompts + 1, dtype=torch.int32, device=device) * prompt_len
    lens = torch.full((prompts,), prompt_len, dtype=torch.int32, device=device)
    owners = torch.arange(prompts, dtype=torch.int32, device=device).repeat_interleave(prompt_len)
    flat = torch.arange(prompt_len, dtype=torch.int32, device=device).repeat(prompts)
    slots = torch.arange(max(batch, prompts), dtype=torch.int32, device=device)

    # Attention, both over the same window.
    query, latent_out = bf16(batch, heads, mixer.row), bf16(batch, heads, KV_RANK)
    t_query, t_out = bf16(tokens, t_heads, t_dim), bf16(tokens, t_heads, t_dim)
    t_key = tide._attention[0][0]
    common = dict(window=window, status=ripe.status)

    def planned(attend):
        """Calls that use the step's work plan, as every layer of a geometry but the first does."""

        attend(False, 0)
        slots_used = iter(range(1, 64))
        return lambda: attend(True, next(slots_used))

    def t_attend(plan, slot):
        sink_decode_attention(t_query[:batch], t_out[:batch], tide.key_blocks[0], tide.value_blocks[0], tables, lengths,
                              scale=0.1, sinks=t.sinks, scratch=tide._scratch[t_key], use_plan=plan, plan_slot=slot, **common)

    def attend(pool, tab, lens, window, scratch):
        return lambda plan, slot: latent_decode_attention(query, latent_out, pool, tab, lens, scale=0.1, sinks=w.sinks,
                                                          window=window, scratch=scratch, use_plan=plan, status=ripe.status)

    def t_prefill():
        sink_prefill_attention(t_query, t_out, tide.key_blocks[0], tide.value_blocks[0], tables_p, cu, lens,
                               max_query_len=prompt_len, scale=0.1, sinks=t.sinks, **common)

    t_decode_work = {"bytes_": batch * reach * kv * t_dim * 4}
    t_prefill_work = {"flops": 4 * t_heads * t_dim * inside}
    def latent_work(seen):
        return {"bytes_": batch * seen * mixer.row * 2, "flops": 2 * heads * batch * seen * (mixer.row + KV_RANK)}

    pair("decode attention", planned(attend(ripe.latents[0], tables, lengths, window, ripe._scratch[ripe._streams[0][0]])),
         planned(t_attend), work=latent_work(reach), their_work=t_decode_work)
    # The same bytes as the other design's window: a cached row is that much smaller.
    equal = t_decode_work["bytes_"] // (batch * mixer.row * 2)
    deep = torch.randn(batch * -(-equal // page), 1, page, mixer.row, device=device).to(torch.bfloat16)
    pair("decode attention, equal bytes", planned(attend(
        deep, _tables(batch, -(-equal // page), deep.shape[0], device), torch.full_like(lengths, equal), None,
        latent_decode_scratch(batch, heads, KV_RANK, batch * equal, device))), planned(t_attend),
        work=latent_work(equal), their_work=t_decode_work)
    del deep
    spans = VisibleSpans(cu, lens, window=window, tokens=tokens, max_query_len=prompt_len, max_context=prompt_len,
                         chunk_starts=[0] * prompts, status=ripe.status)
    rows = spans.gather(ripe.latents[0], tables_p)
    both = ripe._linear(rows, w.expand)
    q_p, out_p = bf16(tokens, heads, mixer.qk_dim), bf16(tokens, heads, HEAD)
    keys, vals = spans.pages(both, 0, heads, mixer.qk_dim), spans.pages(both, heads * mixer.qk_dim, heads, HEAD)
    pair("prefill attention", lambda: sink_prefill_attention(
        q_p, out_p, keys, vals, spans.table, cu, spans.lens, max_query_len=prompt_len, scale=0.1, sinks=w.sinks, **common),
        t_prefill, work={"flops": 2 * heads * (mixer.qk_dim + HEAD) * inside}, their_work=t_prefill_work)
    t_qkv = bf16(tokens, t.qkv.shape[0])

    def t_glue(n, pos, own, tab):
        return lambda: qkv_norm_mix_write(t_qkv[:n], t_query[:n], tide.key_blocks[0], tide.value_blocks[0], pos, own, tab,
                                          q_heads=t_heads, kv_heads=kv, dim=t_dim, value_dim=t_dim, unit_norm=True, eps=1e-6,
                                          v_first=t_qkv[:n, (t_heads + kv) * t_dim:], lam=0.5, status=tide.status)

    pair("prefill gather", lambda: spans.gather(ripe.latents[0], tables_p), t_glue(tokens, flat, owners, tables_p),
         work={"bytes_": 4 * spans.rows * mixer.row}, their_work={"bytes_": 4 * tokens * t.qkv.shape[0]})

    # Recurrent mixers beside attention, then everything that is a pass over rows, then products.
    for label, n, pos, own, tab in (("decode", batch, lengths - 1, None, tables), ("prefill", tokens, flat, owners, tables_p)):
        chunk = {} if label == "decode" else {"cu_seqlens": cu, "max_query_len": prompt_len}
        t_mix, attend_work = (planned(t_attend), t_decode_work) if label == "decode" else (t_prefill, t_prefill_work)
        requests = batch if label == "decode" else prompts
        state_bytes = 4 * (2 if label == "decode" else 1) * requests  # chunks that start at position 0 only write it
        o_rows, o_out = bf16(n, outer.inputs.shape[0]), bf16(n, values)
        pair(f"{label} outer recurrence", lambda: outer_recurrence(
            o_rows, o_out, outer.decay, ripe.state.layer(0), slots[:requests], pos, heads=heads, dim=HEAD, value_dim=HEAD,
            status=ripe.status, **chunk), t_mix,
            work={"bytes_": state_bytes * heads * HEAD * HEAD + 2 * n * 4 * values}, their_work=attend_work)
        a_rows, a_out = bf16(n, 3 * width), bf16(n, width)
        t_act = bf16(n, 2 * ff)
        gate_work = {"bytes_": n * ff * 6}
        pair(f"{label} gated average", lambda: gated_average(
            a_rows, a_out, average.z_bias, average.u_bias, ripe.state.layer(2), slots[:requests], pos, width=width,
            status=ripe.status, **chunk), lambda: clamped_glu(t_act, limit=7.0, slope=1.702, up_offset=1.0),
            work={"bytes_": state_bytes * width + 2 * n * 4 * width}, their_work=gate_work)
        x32, y = torch.randn(n, width, device=device), bf16(n, width)
        norm_work = {"bytes_": n * width * 12}

        def t_norm():
            sum_rms_norm(x32, y, t.norm1, eps=1e-6, alpha=2.0, weight_offset=1.0)

        pair(f"{label} norm + residual + norm", lambda: residual_norm_(x32, y, w.norm1b, w.norm2, alpha=0.5, eps=1e-6),
             t_norm, work=norm_work)
        pair(f"{label} gated norm", lambda: gated_rms_norm(o_out, o_rows[:, -values:], outer.norm, eps=1e-6), t_norm,
             work={"bytes_": n * values * 6}, their_work=norm_work)
        act, side, ids = bf16(n, ff), bf16(n, SIDE), torch.randint(0, vocab, (n,), device=device)
        pair(f"{label} gelu", lambda: gelu(act), lambda: clamped_glu(t_act, limit=7.0, slope=1.702, up_offset=1.0),
             work={"bytes_": n * ff * 4}, their_work=gate_work)
        pair(f"{label} gelu x token rows", lambda: gelu(side, ids=ids, table=w.side_table, status=ripe.status), t_norm,
             work={"bytes_": n * SIDE * 6}, their_work=norm_work)
        down = bf16(n, w.down.shape[0])
        pair(f"{label} latent norms, rotation, page write", lambda: latent_norm_write(
            down, w.q_norm, w.kv_norm, w.turns, ripe.latents[0], pos, own, tab, q_rank=q_rank, rank=KV_RANK,
            rot_dim=ROTATED, rotated=ROTATED, eps=1e-6, status=ripe.status), t_glue(n, pos, own, tab),
            work={"bytes_": 4 * n * w.down.shape[0]}, their_work={"bytes_": 4 * n * t.qkv.shape[0]})
        turned = q_p[:n, :, HEAD:]
        pair(f"{label} query rotation", lambda: rotate_heads(turned, turned, pos, w.turns, ROTATED), t_glue(n, pos, own, tab),
             work={"bytes_": 4 * n * heads * ROTATED}, their_work={"bytes_": 4 * n * t.qkv.shape[0]})
        pair(f"{label} embedding", lambda: embed_tokens(
            ids, ripe.weights.embed, pos, own, tab, scale=2.0, page=page, num_pages=ripe.total_pages, keep_rows=False,
            status=ripe.status), lambda: embed_tokens(
            ids, tide.weights.embed, pos, own, tab, scale=2.0, page=page, num_pages=tide.total_pages,
            bigram=tide.weights.bigram, mul_prev=8191, mul_cur=127, history=tide.history, turns=tide.weights.turns,
            status=tide.status), work={"bytes_": n * width * 6}, their_work={"bytes_": n * width * 10})

        def product(name, x, weight, theirs):
            (k, m), (tk, tm) = (x.shape[1], weight.shape[0]), (theirs.shape[1], theirs.shape[0])
            tx = bf16(x.shape[0], tk)
            pair(f"{label} {name} projection", lambda: ripe._linear(x, weight), lambda: tide._linear(tx, theirs),
                 work={"bytes_": 2 * (m * k + x.shape[0] * (m + k)), "flops": 2 * x.shape[0] * m * k},
                 their_work={"bytes_": 2 * (tm * tk + tx.shape[0] * (tm + tk)), "flops": 2 * tx.shape[0] * tm * tk})

        product("latent down", y, w.down, t.qkv)
        product("query up", bf16(n, q_rank), w.uq, t.qkv)
        product("o", bf16(n, values), w.o, t.o)
        product("recurrent input", y, outer.inputs, t.qkv)
        product("up", y, w.up, t.gate_up)
        product("down", act, w.down_ff, t.down)
        product("side gate", y, w.side_gate, t.o)
        product("side", side, w.side_proj, t.o)
        if label == "prefill":
            product("key / value expansion", rows, w.expand, t.qkv)
        else:
            nope = q_p[:n, :, :HEAD].transpose(0, 1)
            into = query[..., :KV_RANK].transpose(0, 1)
            small = bf16(n, t.o.shape[1])
            o_work = {"bytes_": 2 * (t.o.numel() + n * sum(t.o.shape)), "flops": 2 * n * t.o.numel()}
            up_work = {"bytes_": 2 * heads * (HEAD * KV_RANK + n * (HEAD + KV_RANK)), "flops": 2 * n * heads * HEAD * KV_RANK}
            pair("decode into the latent space", lambda: torch.bmm(nope, w.uk, out=into), lambda: tide._linear(small, t.o),
                 work=up_work, their_work=o_work)
            back = out_p[:n].transpose(0, 1)
            pair("decode out of the latent space", lambda: torch.bmm(latent_out.transpose(0, 1), w.uv.transpose(1, 2), out=back),
                 lambda: tide._linear(small, t.o), work=up_work, their_work=o_work)
        del o_rows, o_out, a_rows, a_out, t_act, x32, y, act
    final = bf16(batch, width)
    pair("lm_head + greedy", lambda: ripe.lm_head_argmax(final, ripe.weights.head),
         lambda: tide.lm_head_argmax(final, tide.weights.head), work={"bytes_": 2 * vocab * width})
    ripe.check_status()
    tide.check_status()
    return out


def run_ripesun(device, hbm: float, tensor: float, *, sizes=tuple(RIPESUN_SIZES), batch: int = 64, context: int = 2048,
                prompts: int = 8, prompt_len: int = 2048, steps: int = 50) -> dict:
    result = {"layers": 8, "window": WINDOW, "decode_batch": batch, "decode_context": context,
              "prefill": f"{prompts} x {prompt_len}", "hbm_gb_s": hbm, "bf16_tflop_s": tensor, "sizes": {}}
    for name in sizes:
        width, heads, ff, q_rank, vocab = size = RIPESUN_SIZES[name]
        pages = max(batch * (-(-(context + steps + 16) // 16)), prompts * (-(-prompt_len // 16))) + 8
        options = dict(num_pages=pages, max_batch=batch, max_context=context + steps + 64, kv_init="normal")
        ripe = RipesunRunner(RipesunWeights.random(RipesunShape.from_config(ripesun_config(*size)), device), **options)
        entry = {"ripesun": _throughput(ripe, vocab, batch, context, prompts, prompt_len, steps, device)}
        one = _throughput(ripe, vocab, 1, context, 1, prompt_len, steps, device)
        entry["ripesun, one request"] = one
        ripe.release_graphs()
        tide_shape = TidelornShape.from_config(tidelorn_config(width, heads, heads // 2, HEAD, ff, vocab, windowed_only=True))
        tide = TidelornRunner(TidelornWeights.random(tide_shape, device), **options)
        entry["tidelorn"] = _throughput(tide, vocab, batch, context, prompts, prompt_len, steps, device)
        entry["tidelorn, one request"] = _throughput(tide, vocab, 1, context, 1, prompt_len, steps, device)
        tide.release_graphs()
        entry["kernels"] = _ripesun_kernels(size, ripe, tide, batch, context, prompts, prompt_len, hbm, tensor, device)
        result["sizes"][name] = entry
        del ripe, tide
        gc.collect()
        torch.cuda.empty_cache()
    return result

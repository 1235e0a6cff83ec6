"""The Ripesun decoder on the paged step machinery.

A decoder with a 32-bit residual stream whose layers have one of three mixers, each sublayer normed before and after,
and a per-layer token input:

  x <- x + m norm1b(mixer(norm1(x)));  x <- x + m norm2b(ff(norm2(x)));  x <- x + m side_norm(side(x, token))

Mixers: latent attention (queries and keys / values through low-rank latents, a rotated key part shared by the heads,
a sliding window, a sink per head; a layer may read an earlier layer's cached rows), decayed outer products per head
("lightning"), a gated average per channel ("mingru").  Logits are soft-capped.

Cache: every latent layer that projects its own rows has a pool ``[pages, 1, page, kv_rank + rot_dim]`` under the
shared block tables.  State: the recurrent layers' fp32 state is one row of ``StateBuffer`` per request, named by the
step's ``state_slots``.

One latent layer is

  merged query / key-value down projection -> norms, rotation, page write -> query up projection ->
    single tokens:  queries into the latent space, attention over the cached rows, values out of it
    prompt chunks:  visible rows gathered and projected to heads, tcgen05 attention
  -> o projection

and a recurrent layer one merged projection, the recurrence, (norm and gate,) and the o projection; between sublayers
one kernel norms the result, adds it to the residual stream and norms the stream for what comes next.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from types import SimpleNamespace

import torch

from ..kernels.decoder_glue import (
    embed_tokens,
    gated_rms_norm,
    gelu,
    residual_norm_,
    sinusoid_turns,
    softcap_,
    sum_rms_norm,
)
from ..kernels.recurrence import StateBuffer, gated_average, outer_recurrence
from ..kv_cache.latent_attention import (
    VisibleSpans,
    latent_decode_attention,
    latent_decode_scratch,
    latent_decode_supported,
    latent_norm_write,
    rotate_heads,
)
from ..kv_cache.sink_attention import attention_rows, sink_prefill_attention, sink_prefill_supported
from ... import _lib
from .step_runner import PagedStepRunner


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int                # unrotated query / key entries per head
    rot_dim: int            # query / key entries per head that carry positions; the key's are shared by the heads
    rotated: int            # of those, how many are rotated
    rot_base: float
    vdim: int
    q_rank: int
    kv_rank: int
    window: int
    scale: float
    kv_from: int | None     # layer whose cached rows this one reads; None: its own

    @property
    def row(self) -> int:
        """Entries of a cached row."""

        return self.kv_rank + self.rot_dim

    @property
    def qk_dim(self) -> int:
        return self.dim + self.rot_dim

    def tensor_shapes(self, width: int) -> dict[str, tuple[int, ...]]:
        out = {"dq": (self.q_rank, width), "dq.norm": (self.q_rank,), "uq": (self.heads * self.qk_dim, self.q_rank)}
        if self.kv_from is None:
            out["dkv"], out["dkv.norm"] = (self.row, width), (self.kv_rank,)
        out["uk"], out["uv"] = (self.heads * self.dim, self.kv_rank), (self.heads * self.vdim, self.kv_rank)
        out["sink"], out["o"] = (self.heads,), (width, self.heads * self.vdim)
        return out


@dataclass(frozen=True)
class OuterMixer:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    @property
    def state_floats(self) -> int:
        return self.heads * self.dim * self.vdim

    def tensor_shapes(self, width: int) -> dict[str, tuple[int, ...]]:
        keys, values = self.heads * self.dim, self.heads * self.vdim
        return {"q": (keys, width), "k": (keys, width), "v": (values, width), "g": (values, width),
                "o": (width, values), "norm": (values,)}


@dataclass(frozen=True)
class AverageMixer:
    width: int

    @property
    def state_floats(self) -> int:
        return self.width

    def tensor_shapes(self, width: int) -> dict[str, tuple[int, ...]]:
        return {"z": (self.width, width), "z.b": (self.width,), "x": (self.width, width), "x.b": (self.width,),
                "g": (self.width, width), "o": (width, self.width)}


@dataclass(frozen=True)
class RipesunLayer:
    mixer: LatentMixer | OuterMixer | AverageMixer
    ff: int | None          # None: no feed-forward (and no norms around it)


def _latent_mixer(mixer: dict) -> LatentMixer:
    return LatentMixer(
        heads=int(mixer["heads"]), dim=int(mixer["dim"]), rot_dim=int(mixer["rot_dim"]),
        rotated=int(mixer["rot"]["dims"]), rot_base=float(mixer["rot"]["base"]), vdim=int(mixer["vdim"]),
        q_rank=int(mixer["q_rank"]), kv_rank=int(mixer["kv_rank"]), window=int(mixer["mask"]["size"]),
        scale=float(mixer["scale"]), kv_from=None if mixer.get("kv_from") is None else int(mixer["kv_from"]))


def _outer_mixer(mixer: dict) -> OuterMixer:
    return OuterMixer(heads=int(mixer["heads"]), dim=int(mixer["dim"]), vdim=int(mixer["vdim"]),
                      decay=tuple(float(d) for d in mixer["decay"]))


MIXERS = {"latent_attention": _latent_mixer, "lightning": _outer_mixer,
          "mingru": lambda mixer: AverageMixer(int(mixer["width"]))}


@dataclass(frozen=True)
class RipesunShape:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    embed_scale: float
    side_dim: int
    logit_softcap: float
    layers: tuple[RipesunLayer, ...]
    page: int = 16

    @classmethod
    def from_config(cls, config: dict, page: int = 16) -> "RipesunShape":
        layers: list[RipesunLayer] = []
        for index, entry in enumerate(config["layers"]):
            kind, mlp = entry["type"], entry.get("mlp")
            if kind not in MIXERS:
                raise ValueError(f"layer {index}: unknown type {kind!r}")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {index}: unknown feed-forward {mlp['kind']!r}")
            mixer = MIXERS[kind](entry["mixer"])
            if isinstance(mixer, LatentMixer):
                if mixer.window < 1:
                    raise ValueError(f"layer {index}: the window must be positive")
                if mixer.rotated % 2 or not 0 <= mixer.rotated <= mixer.rot_dim:
                    raise ValueError(f"layer {index}: an even number of at most rot_dim entries is rotated")
                if mixer.kv_from is not None:
                    source = layers[mixer.kv_from].mixer if 0 <= mixer.kv_from < index else None
                    if not isinstance(source, LatentMixer) or source.kv_from is not None:
                        raise ValueError(f"layer {index}: kv_from must name an earlier layer with cached rows of its own")
                    same = ("kv_rank", "rot_dim", "rotated", "rot_base")
                    if any(getattr(source, name) != getattr(mixer, name) for name in same):
                        raise ValueError(f"layer {index}: kv_from needs equal kv_rank, rot_dim and rotation")
            if isinstance(mixer, OuterMixer) and len(mixer.decay) != mixer.heads:
                raise ValueError(f"layer {index}: one decay per head")
            layers.append(RipesunLayer(mixer, None if mlp is None else int(mlp["ff"])))
        return cls(vocab=int(config["vocab"]), width=int(config["width"]), eps=float(config["norm"]["eps"]),
                   residual_mult=float(config["residual_mult"]), embed_scale=float(config["embedding"]["scale"]),
                   side_dim=int(config["token_side"]["dim"]), logit_softcap=float(config["logit_softcap"]),
                   layers=tuple(layers), page=page)

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Name and shape of every tensor of a checkpoint."""

        out = {"embed": (self.vocab, self.width), "side.embed": (self.vocab, len(self.layers) * self.side_dim)}
        for i, layer in enumerate(self.layers):
            out[f"l{i}.norm1"] = out[f"l{i}.norm1b"] = (self.width,)
            for name, size in layer.mixer.tensor_shapes(self.width).items():
                out[f"l{i}.mix.{name}"] = size
            if layer.ff is not None:
                out[f"l{i}.norm2"] = out[f"l{i}.norm2b"] = (self.width,)
                out[f"l{i}.mlp.up"], out[f"l{i}.mlp.down"] = (layer.ff, self.width), (self.width, layer.ff)
            out[f"l{i}.side.gate"], out[f"l{i}.side.proj"] = (self.side_dim, self.width), (self.width, self.side_dim)
            out[f"l{i}.side.norm"] = (self.width,)
        out["final.norm"], out["head"] = (self.width,), (self.vocab, self.width)
        return out


class RipesunWeights:
    """Weights in the form the runner uses, everything in ``dtype`` except sinks, decays and rotation turns (fp32).

    Projections of the same input are merged: query and key / value down projection (``down``), the recurrent mixers'
    inputs (``inputs``).  ``expand`` maps a cached row to every head's [key | rotated part] and then to the values: the
    rotated part goes through an identity block, so one product makes whole keys.  ``uk`` and ``uv`` are the same
    up projections per head, for the absorbed form."""

    def __init__(self, shape: RipesunShape, take, device: torch.device, dtype: torch.dtype = torch.bfloat16) -> None:
        """``take(name, shape)`` returns a checkpoint tensor."""

        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("weights are bfloat16 or float32")
        self.shape, self.device, self.dtype = shape, device, dtype
        shapes = shape.tensor_shapes()

        def fetch(name: str, kind: torch.dtype = dtype) -> torch.Tensor:
            return take(name, shapes[name]).to(device=device, dtype=kind).contiguous()

        self.embed, self.side_embed = fetch("embed"), fetch("side.embed")
        self.layers: list[SimpleNamespace] = []
        for i, layer in enumerate(shape.layers):
            prefix = f"l{i}."
            w = SimpleNamespace(
                norm1=fetch(prefix + "norm1"), norm1b=fetch(prefix + "norm1b"), o=fetch(prefix + "mix.o"),
                norm2=None, norm2b=None, up=None, down_ff=None,
                side_gate=fetch(prefix + "side.gate"), side_proj=fetch(prefix + "side.proj"),
                side_norm=fetch(prefix + "side.norm"),
                side_table=self.side_embed[:, i * shape.side_dim:(i + 1) * shape.side_dim])
            if layer.ff is not None:
                w.norm2, w.norm2b = fetch(prefix + "norm2"), fetch(prefix + "norm2b")
                w.up, w.down_ff = fetch(prefix + "mlp.up"), fetch(prefix + "mlp.down")
            mix = prefix + "mix."
            if isinstance(layer.mixer, LatentMixer):
                self._latent(w, layer.mixer, lambda name, *kind: fetch(mix + name, *kind))
            elif isinstance(layer.mixer, OuterMixer):
                w.inputs = torch.cat([fetch(mix + name) for name in "qkvg"])
                w.norm = fetch(mix + "norm")
                w.decay = torch.tensor(layer.mixer.decay, dtype=torch.float32, device=device)
            else:
                w.inputs = torch.cat([fetch(mix + name) for name in "zxg"])
                w.z_bias, w.u_bias = fetch(mix + "z.b"), fetch(mix + "x.b")
            self.layers.append(w)
        self.final_norm, self.head = fetch("final.norm"), fetch("head")

    def _latent(self, w: SimpleNamespace, mixer: LatentMixer, fetch) -> None:
        own = mixer.kv_from is None
        w.down = torch.cat([fetch("dq"), fetch("dkv")]) if own else fetch("dq")
        w.q_norm, w.kv_norm = fetch("dq.norm"), fetch("dkv.norm") if own else None
        w.uq, w.sinks = fetch("uq"), fetch("sink", torch.float32)
        w.uk = fetch("uk").view(mixer.heads, mixer.dim, mixer.kv_rank)
        w.uv = fetch("uv").view(mixer.heads, mixer.vdim, mixer.kv_rank)
        keys = torch.zeros(mixer.heads, mixer.qk_dim, mixer.row, dtype=self.dtype, device=self.device)
        keys[:, :mixer.dim, :mixer.kv_rank] = w.uk
        keys[:, mixer.dim:, mixer.kv_rank:] = torch.eye(mixer.rot_dim, dtype=self.dtype, device=self.device)
        values = torch.zeros(mixer.heads * mixer.vdim, mixer.row, dtype=self.dtype, device=self.device)
        values[:, :mixer.kv_rank] = w.uv.reshape(mixer.heads * mixer.vdim, mixer.kv_rank)
        w.expand = torch.cat([keys.view(mixer.heads * mixer.qk_dim, mixer.row), values])
        w.turns = sinusoid_turns(mixer.rotated, mixer.rot_base, self.device) if mixer.rotated else None

    @classmethod
    def random(cls, shape: RipesunShape, device: torch.device, *, seed: int = 0,
               dtype: torch.dtype = torch.bfloat16) -> "RipesunWeights":
        """Seeded random weights of the checkpoint's form (drawn on ``device``)."""

        generator = torch.Generator(device=device).manual_seed(seed)

        def take(name: str, size: tuple[int, ...]) -> torch.Tensor:
            noise = torch.randn(size, generator=generator, device=device, dtype=torch.float32)
            if "norm" in name:
                noise = noise.mul(0.1).add(1.0)
            elif name.endswith((".b", "sink")):
                noise = noise * 0.5
            elif name not in ("embed", "side.embed"):
                noise = noise / math.sqrt(size[1])
            return noise.to(torch.bfloat16)

        return cls(shape, take, device, dtype)

    def weight_bytes(self) -> int:
        """Bytes a decode step streams (projections and head; the embedding rows are a few)."""

        total = self.head.numel()
        for w in self.layers:
            names = ("o", "up", "down_ff", "side_gate", "side_proj", "inputs", "down", "uq", "uk", "uv")
            total += sum(t.numel() for t in (getattr(w, n, None) for n in names) if t is not None)
        return total * self.dtype.itemsize


class RipesunRunner(PagedStepRunner):
    """Steps of a Ripesun model over its latent pages and state slots (pages, buckets and graphs:
    ``PagedStepRunner``)."""

    wants_chunk_starts = True

    def __init__(self, weights: RipesunWeights, *, num_pages: int, max_batch: int, max_context: int,
                 decode_buckets: tuple[int, ...] | None = None, chunk_buckets: tuple[int, ...] = (128, 512),
                 max_chunks: int = 4, state_slots: int | None = None, kv_init: str = "zeros",
                 attention: str = "auto") -> None:
        """``state_slots``: requests that can be live at once (default ``max_batch``; more lets a prefix cache keep
        states).  ``attention``: "auto" takes the streaming kernels where a layer's sizes and number format allow
        them, "rows" the row kernel everywhere."""

        if attention not in ("auto", "rows"):
            raise ValueError("attention must be 'auto' or 'rows'")
        super().__init__(weights.shape, weights.device, num_pages=num_pages, max_batch=max_batch,
                         max_context=max_context, decode_buckets=decode_buckets, chunk_buckets=chunk_buckets,
                         max_chunks=max_chunks, state_slots=max_batch if state_slots is None else state_slots)
        self.weights, self.dtype = weights, weights.dtype
        # Library products accumulate in full fp32: no TF32 for fp32 operands, no bf16 partial sums for bf16 ones.
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        layers, page = self.shape.layers, self.shape.page
        self.latents: list[torch.Tensor | None] = []
        self._state_index: dict[int, int] = {}
        sizes: list[int] = []
        # Layers of one geometry share a split-KV work plan within a step, and its scratch.
        self._streams: list[tuple[tuple, bool, bool] | None] = []  # (plan key, streams decode rows, expands chunks)
        self._scratch: dict[tuple, torch.Tensor] = {}
        rows = max(max_batch, self.decode_buckets[-1])
        for index, layer in enumerate(layers):
            mixer, pool, streams = layer.mixer, None, None
            if isinstance(mixer, LatentMixer):
                if mixer.kv_from is None:
                    pool = torch.zeros(self.total_pages, 1, page, mixer.row, dtype=self.dtype, device=self.device)
                    if kv_init == "normal":
                        pool.normal_()
                decode = attention == "auto" and latent_decode_supported(mixer.row, mixer.kv_rank, page, self.dtype)
                chunks = attention == "auto" and sink_prefill_supported(
                    mixer.heads, mixer.heads, mixer.qk_dim, mixer.vdim, 16, self.dtype, mixer.scale)
                key = (mixer.heads, mixer.row, mixer.kv_rank, mixer.window)
                if decode and key not in self._scratch:
                    reach = min(max_context, mixer.window + 16)
                    self._scratch[key] = latent_decode_scratch(rows, mixer.heads, mixer.kv_rank, rows * reach,
                                                               self.device)
                streams = (key, decode, chunks)
            else:
                self._state_index[index] = len(sizes)
                sizes.append(mixer.state_floats)
            self.latents.append(pool)
            self._streams.append(streams)
        self.state = StateBuffer(sizes, self.total_slots, self.device)

    def copy_state(self, source: int, target: int) -> None:
        """Copy a request's whole recurrent state to another slot."""

        self.state.copy(source, target)

    # -- projections ----------------------------------------------------------------------------

    @staticmethod
    def _linear(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
        return torch.nn.functional.linear(x, weight)

    def _finish(self, x32: torch.Tensor, return_logits: bool):
        """Final norm, then greedy tokens (and the logits when asked for) of residual rows.  The soft cap is monotonic:
        the fused head takes the maximum of the logits before it."""

        weights = self.weights
        _, final = sum_rms_norm(x32, None, weights.final_norm, eps=self.shape.eps, keep32=False)
        if not return_logits and self.can_fuse_lm_head(final, weights.head):
            return self.lm_head_argmax(final, weights.head)
        head = weights.head.t()
        logits = torch.mm(final, head) if self.dtype == torch.float32 else torch.mm(final, head, out_dtype=torch.float32)
        tokens = logits.argmax(dim=-1)
        return (tokens, softcap_(logits, self.shape.logit_softcap)) if return_logits else tokens

    # -- mixers ---------------------------------------------------------------------------------

    def _latent_attention(self, index: int, h: torch.Tensor, step: SimpleNamespace) -> torch.Tensor:
        mixer, w = self.shape.layers[index].mixer, self.weights.layers[index]
        source = index if mixer.kv_from is None else mixer.kv_from
        pages, tokens = self.latents[source], int(h.shape[0])
        compressed = latent_norm_write(
            self._linear(h, w.down), w.q_norm, w.kv_norm, w.turns, pages if source == index else None, step.positions,
            step.token_to_sequence, step.block_tables, q_rank=mixer.q_rank, rank=mixer.kv_rank, rot_dim=mixer.rot_dim,
            rotated=mixer.rotated, eps=self.shape.eps, status=self.status)
        q = self._linear(compressed, w.uq).view(tokens, mixer.heads, mixer.qk_dim)
        attended = torch.empty(tokens, mixer.heads, mixer.vdim, dtype=self.dtype, device=self.device)
        expands = tokens > step.decode_rows and self._streams[index][2]
        absorbed = step.decode_rows if expands else tokens
        if absorbed:
            self._absorbed(index, q[:absorbed], attended[:absorbed], pages, step)
        if expands:
            self._expanded(index, source, q[step.decode_rows:], attended[step.decode_rows:], step)
        return self._linear(attended.view(tokens, mixer.heads * mixer.vdim), w.o)

    def _absorbed(self, index: int, q, attended, pages, step: SimpleNamespace) -> None:
        """Attention in the latent space, the leading ``decode_rows`` rows and what the expanded form does not take."""

        mixer, w = self.shape.layers[index].mixer, self.weights.layers[index]
        rows = int(q.shape[0])
        query = torch.empty(rows, mixer.heads, mixer.row, dtype=self.dtype, device=self.device)
        torch.bmm(q[..., :mixer.dim].transpose(0, 1), w.uk, out=query[..., :mixer.kv_rank].transpose(0, 1))
        rotate_heads(q[..., mixer.dim:], query[..., mixer.kv_rank:], step.positions, w.turns, mixer.rotated)
        out = torch.empty(rows, mixer.heads, mixer.kv_rank, dtype=self.dtype, device=self.device)
        common = dict(scale=mixer.scale, window=mixer.window, sinks=w.sinks, status=self.status)
        key, streams, _ = self._streams[index]
        single = step.decode_rows if streams else 0
        if single:
            latent_decode_attention(query[:single], out[:single], pages, step.block_tables[:single],
                                    step.decode_lengths, scratch=self._scratch[key], use_plan=key in step.plans, **common)
            step.plans.add(key)
        if rows > single:
            part = slice(single, rows)
            owners = None if step.token_to_sequence is None else step.token_to_sequence[part]
            attention_rows(query[part], out[part], pages, pages[..., :mixer.kv_rank], step.positions[part], owners,
                           step.block_tables, **common)
        torch.bmm(out.transpose(0, 1), w.uv.transpose(1, 2), out=attended.transpose(0, 1))

    def _expanded(self, index: int, source: int, q, attended, step: SimpleNamespace) -> None:
        """Packed chunks over per-head keys and values of the cached rows they see."""

        mixer, w = self.shape.layers[index].mixer, self.weights.layers[index]
        rotated = q[..., mixer.dim:]
        rotate_heads(rotated, rotated, step.positions[step.decode_rows:], w.turns, mixer.rotated)
        spans = step.spans.get(mixer.window)
        if spans is None:
            spans = step.spans[mixer.window] = VisibleSpans(
                step.cu_seqlens, step.kv_lens, window=mixer.window, tokens=int(q.shape[0]),
                max_query_len=step.max_query_len, max_context=self.max_context, chunk_starts=step.chunk_starts,
                status=self.status)
        rows = step.gathered.get((source, mixer.window))
        if rows is None:
            rows = step.gathered[source, mixer.window] = spans.gather(self.latents[source],
                                                                      step.block_tables[step.decode_rows:])
        both = self._linear(rows, w.expand)
        keys = spans.pages(both, 0, mixer.heads, mixer.qk_dim)
        values = spans.pages(both, mixer.heads * mixer.qk_dim, mixer.heads, mixer.vdim)
        sink_prefill_attention(q, attended, keys, values, spans.table, step.cu_seqlens, spans.lens,
                               max_query_len=step.max_query_len, scale=mixer.scale, window=mixer.window, sinks=w.sinks,
                               status=self.status)

    def _recurrent(self, index: int, run, rows: torch.Tensor, out: torch.Tensor, step: SimpleNamespace, *arguments,
                   **sizes) -> None:
        """``run`` on the single tokens and on the packed chunks of a step."""

        state, single = self.state.layer(self._state_index[index]), step.decode_rows
        if single:
            run(rows[:single], out[:single], *arguments, state, step.state_slots[:single], step.positions[:single],
                status=self.status, **sizes)
        if rows.shape[0] > single:
            run(rows[single:], out[single:], *arguments, state, step.state_slots[single:], step.positions[single:],
                cu_seqlens=step.cu_seqlens, max_query_len=step.max_query_len, status=self.status, **sizes)

    def _lightning(self, index: int, h: torch.Tensor, step: SimpleNamespace) -> torch.Tensor:
        mixer, w = self.shape.layers[index].mixer, self.weights.layers[index]
        values = mixer.heads * mixer.vdim
        rows = self._linear(h, w.inputs)
        out = torch.empty(int(h.shape[0]), values, dtype=self.dtype, device=self.device)
        self._recurrent(index, outer_recurrence, rows, out, step, w.decay, heads=mixer.heads, dim=mixer.dim,
                        value_dim=mixer.vdim)
        return self._linear(gated_rms_norm(out, rows[:, -values:], w.norm, eps=self.shape.eps), w.o)

    def _mingru(self, index: int, h: torch.Tensor, step: SimpleNamespace) -> torch.Tensor:
        mixer, w = self.shape.layers[index].mixer, self.weights.layers[index]
        rows = self._linear(h, w.inputs)
        out = torch.empty(int(h.shape[0]), mixer.width, dtype=self.dtype, device=self.device)
        self._recurrent(index, gated_average, rows, out, step, w.z_bias, w.u_bias, width=mixer.width)
        return self._linear(out, w.o)

    # -- the layers -----------------------------------------------------------------------------

    def _layers(self, input_ids, positions, token_to_sequence, block_tables, *, state_slots, decode_rows: int,
                decode_lengths, cu_seqlens=None, kv_lens=None, max_query_len: int = 0, chunk_starts=None) -> torch.Tensor:
        """Residual rows after the last layer (fp32), cache and state holding the new tokens."""

        shape, weights = self.shape, self.weights
        step = SimpleNamespace(positions=positions, token_to_sequence=token_to_sequence, block_tables=block_tables,
                               state_slots=state_slots, decode_rows=decode_rows, decode_lengths=decode_lengths,
                               cu_seqlens=cu_seqlens, kv_lens=kv_lens, max_query_len=max_query_len,
                               chunk_starts=chunk_starts, plans=set(), spans={}, gathered={})
        mixers = {LatentMixer: self._latent_attention, OuterMixer: self._lightning, AverageMixer: self._mingru}
        x32, _ = embed_tokens(input_ids, weights.embed, positions, token_to_sequence, block_tables,
                              scale=shape.embed_scale, page=shape.page, num_pages=self.total_pages, keep_rows=False,
                              status=self.status)
        _, h = sum_rms_norm(x32, None, weights.layers[0].norm1, eps=shape.eps, keep32=False)
        add = dict(alpha=shape.residual_mult, eps=shape.eps)
        for index, (layer, w) in enumerate(zip(shape.layers, weights.layers)):
            y = mixers[type(layer.mixer)](index, h, step)
            if layer.ff is not None:
                h = residual_norm_(x32, y, w.norm1b, w.norm2, **add)
                y = self._linear(gelu(self._linear(h, w.up)), w.down_ff)
                x = residual_norm_(x32, y, w.norm2b, **add)
            else:
                x = residual_norm_(x32, y, w.norm1b, **add)
            side = gelu(self._linear(x, w.side_gate), ids=input_ids, table=w.side_table, status=self.status)
            last = index + 1 == len(shape.layers)
            h = residual_norm_(x32, self._linear(side, w.side_proj), w.side_norm,
                               None if last else weights.layers[index + 1].norm1, keep_rows=not last, **add)
        return x32

    # -- the two forwards -----------------------------------------------------------------------

    def decode_forward(self, input_ids: torch.Tensor, sequence_lengths: torch.Tensor, block_tables: torch.Tensor,
                       return_logits: bool = False, *, state_slots: torch.Tensor):
        """One token per block-table row, at position ``length - 1`` (``sequence_lengths`` counts it), row i's state in
        slot ``state_slots[i]``.  Returns the greedy next tokens (int64), with ``return_logits`` also their fp32
        logits."""

        before = _lib.load().mie_launch_count()
        x32 = self._layers(input_ids, sequence_lengths - 1, None, block_tables, state_slots=state_slots,
                           decode_rows=int(input_ids.shape[0]), decode_lengths=sequence_lengths)
        out = self._finish(x32, return_logits)
        self.launches_per_step = int(_lib.load().mie_launch_count() - before)
        return out

    def mixed_forward(self, input_ids: torch.Tensor, token_to_sequence: torch.Tensor, token_positions: torch.Tensor,
                      block_tables: torch.Tensor, *, decode_rows: int, decode_lengths, cu_seqlens: torch.Tensor,
                      kv_lens: torch.Tensor, max_query_len: int, logit_rows: torch.Tensor,
                      return_logits: bool = False, state_slots: torch.Tensor, chunk_starts=None):
        """Decode rows (one per leading block-table row) and packed prompt chunks in one flat stream; the rows in
        ``logit_rows`` are projected to logits.  ``state_slots``: one per block-table row."""

        before = _lib.load().mie_launch_count()
        x32 = self._layers(input_ids, token_positions, token_to_sequence, block_tables, state_slots=state_slots,
                           decode_rows=decode_rows, decode_lengths=decode_lengths, cu_seqlens=cu_seqlens,
                           kv_lens=kv_lens, max_query_len=max_query_len, chunk_starts=chunk_starts)
        out = self._finish(x32.index_select(0, logit_rows), return_logits)
        self.launches_per_step = int(_lib.load().mie_launch_count() - before)
        return out


__all__ = ["AverageMixer", "LatentMixer", "OuterMixer", "RipesunLayer", "RipesunRunner", "RipesunShape",
           "RipesunWeights"]

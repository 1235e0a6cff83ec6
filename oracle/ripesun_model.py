"""Plain, slow restatement of the Ripesun decoder.  TEST INFRASTRUCTURE ONLY.

One function per mechanism, straight from the equations, on dense tensors of one sequence: no pages, no cache, no
batching, no absorbed projections, no chunked recurrences and nothing shared with the product path.  Everything is
computed in the dtype of ``weights`` (float64 by default).  ``config`` is the parsed config.json: ``vocab``,
``width``, ``norm.eps``, ``residual_mult``, ``embedding.scale``, ``token_side.dim``, ``logit_softcap``, ``layers``.

Notation: x [T, width] is the residual stream of one sequence, p = 0 ... T-1 its positions.
"""

from __future__ import annotations

import math

import torch


# -- mechanisms ---------------------------------------------------------------------------------------

def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension, eps under the root."""

    return x / torch.sqrt(x.square().mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * weight


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    """z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))."""

    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rotate(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """Rotary positions on the first ``dims`` entries of the last dimension of x [T, ..., n], entry 2i paired with
    entry 2i + 1 and turned by p * base^(-2i / dims)."""

    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(torch.float64) * base ** (-2.0 * i / dims)
        shape = (-1,) + (1,) * (x.ndim - 2)
        cos, sin = (f(angle).to(x.dtype).view(shape) for f in (torch.cos, torch.sin))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * cos - v * sin
        out[..., 2 * i + 1] = v * cos + u * sin
    return out


def visibility(length: int, window: int) -> torch.Tensor:
    """[T, T]: query i sees key j when 0 <= i - j < window."""

    distance = torch.arange(length).unsqueeze(1) - torch.arange(length).unsqueeze(0)
    return (distance >= 0) & (distance < window)


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum_j exp(s_j)) along the last dimension; ``sink`` broadcasts over rows."""

    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink)
    weights = torch.exp(scores - top)
    return weights / (torch.exp(sink - top) + weights.sum(dim=-1, keepdim=True))


def decayed_outer_products(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: list[float]) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, e] -> o [T, H, e]: S <- decay_h S + k v^T, o = S^T q, token after token."""

    length, heads, _ = q.shape
    out = torch.zeros_like(v)
    for h in range(heads):
        state = torch.zeros(k.shape[2], v.shape[2], dtype=q.dtype)
        for t in range(length):
            state = decay[h] * state + torch.outer(k[t, h], v[t, h])
            out[t, h] = state.t() @ q[t, h]
    return out


def gru_candidate(u: torch.Tensor) -> torch.Tensor:
    """Half a unit above u on the non-negative side, the logistic function on the negative one (both 1/2 at 0)."""

    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def gated_average(z: torch.Tensor, candidate: torch.Tensor) -> torch.Tensor:
    """S <- (1 - z) S + z candidate, element by element, token after token; all S [T, n]."""

    state, out = torch.zeros_like(z[0]), torch.empty_like(z)
    for t in range(z.shape[0]):
        state = (1.0 - z[t]) * state + z[t] * candidate[t]
        out[t] = state
    return out


def softcap(logits: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(logits / cap)


# -- mixers -------------------------------------------------------------------------------------------

def latent_keys(config: dict, weights: dict, index: int, h: torch.Tensor):
    """The normed latent [T, kv_rank] and the rotated shared key part [T, rot_dim] of a layer that projects them."""

    mixer, prefix = config["layers"][index]["mixer"], f"l{index}.mix."
    both = h @ weights[prefix + "dkv"].t()
    rank = mixer["kv_rank"]
    latent = rms_norm(both[:, :rank], weights[prefix + "dkv.norm"], config["norm"]["eps"])
    rotated = rotate(both[:, rank:], torch.arange(h.shape[0]), mixer["rot"]["dims"], mixer["rot"]["base"])
    return latent, rotated


def latent_attention(config: dict, weights: dict, index: int, h: torch.Tensor, latents: dict) -> torch.Tensor:
    """``latents`` maps a layer to its (latent, rotated key part); a layer without ``kv_from`` adds its own."""

    mixer, prefix = config["layers"][index]["mixer"], f"l{index}.mix."
    heads, dim, rot, vdim = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"]
    length = h.shape[0]
    source = mixer.get("kv_from")
    if source is None:
        latents[index] = latent_keys(config, weights, index, h)
        source = index
    latent, shared = latents[source]
    compressed = rms_norm(h @ weights[prefix + "dq"].t(), weights[prefix + "dq.norm"], config["norm"]["eps"])
    q = (compressed @ weights[prefix + "uq"].t()).view(length, heads, dim + rot)
    q_rot = rotate(q[..., dim:], torch.arange(length), mixer["rot"]["dims"], mixer["rot"]["base"])
    k = (latent @ weights[prefix + "uk"].t()).view(length, heads, dim)
    v = (latent @ weights[prefix + "uv"].t()).view(length, heads, vdim)
    seen = visibility(length, mixer["mask"]["size"])
    out = torch.empty(length, heads, vdim, dtype=h.dtype)
    for head in range(heads):
        scores = (q[:, head, :dim] @ k[:, head].t() + q_rot[:, head] @ shared.t()) * mixer["scale"]
        scores = scores.masked_fill(~seen, -math.inf)
        out[:, head] = sink_softmax(scores, weights[prefix + "sink"][head]) @ v[:, head]
    return out.reshape(length, heads * vdim) @ weights[prefix + "o"].t()


def lightning(config: dict, weights: dict, index: int, h: torch.Tensor) -> torch.Tensor:
    mixer, prefix = config["layers"][index]["mixer"], f"l{index}.mix."
    heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
    length = h.shape[0]

    def project(name, size):
        return silu(h @ weights[prefix + name].t()).view(length, heads, size)

    out = decayed_outer_products(project("q", dim), project("k", dim), project("v", vdim), mixer["decay"])
    out = rms_norm(out.reshape(length, heads * vdim), weights[prefix + "norm"], config["norm"]["eps"])
    return (out * torch.sigmoid(h @ weights[prefix + "g"].t())) @ weights[prefix + "o"].t()


def mingru(config: dict, weights: dict, index: int, h: torch.Tensor) -> torch.Tensor:
    prefix = f"l{index}.mix."
    z = torch.sigmoid(h @ weights[prefix + "z"].t() + weights[prefix + "z.b"])
    u = h @ weights[prefix + "x"].t() + weights[prefix + "x.b"]
    states = gated_average(z, gru_candidate(u))
    return (states * silu(h @ weights[prefix + "g"].t())) @ weights[prefix + "o"].t()


# -- the model ----------------------------------------------------------------------------------------

def feed_forward(weights: dict, index: int, h: torch.Tensor) -> torch.Tensor:
    return gelu_tanh(h @ weights[f"l{index}.mlp.up"].t()) @ weights[f"l{index}.mlp.down"].t()


def token_side(config: dict, weights: dict, index: int, x: torch.Tensor, tokens: list[int]) -> torch.Tensor:
    """What the per-layer token input adds to the stream, before the residual multiplier."""

    dim, prefix = config["token_side"]["dim"], f"l{index}.side."
    entry = weights["side.embed"][torch.tensor(tokens), index * dim:(index + 1) * dim]
    y = (gelu_tanh(x @ weights[prefix + "gate"].t()) * entry) @ weights[prefix + "proj"].t()
    return rms_norm(y, weights[prefix + "norm"], config["norm"]["eps"])


def forward(config: dict, weights: dict, tokens: list[int]):
    """``(logits [T, vocab], residual stream after every layer [layers, T, width])`` of one whole sequence."""

    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = weights["embed"][torch.tensor(tokens)] * config["embedding"]["scale"]
    streams, latents = [], {}
    for index, layer in enumerate(config["layers"]):
        h = rms_norm(x, weights[f"l{index}.norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(config, weights, index, h, latents)
        else:
            y = {"lightning": lightning, "mingru": mingru}[layer["type"]](config, weights, index, h)
        x = x + mult * rms_norm(y, weights[f"l{index}.norm1b"], eps)
        if layer["mlp"] is not None:
            y = feed_forward(weights, index, rms_norm(x, weights[f"l{index}.norm2"], eps))
            x = x + mult * rms_norm(y, weights[f"l{index}.norm2b"], eps)
        x = x + mult * token_side(config, weights, index, x, tokens)
        streams.append(x)
    logits = rms_norm(x, weights["final.norm"], eps) @ weights["head"].t()
    return softcap(logits, config["logit_softcap"]), torch.stack(streams)


def greedy(config: dict, weights: dict, prompt: list[int], new_tokens: int):
    """Greedy continuation by recomputing the whole sequence for every token.  Returns ``(tokens, margin)``: the
    smallest top-2 logit gap over the steps divided by the spread of that step's logits."""

    tokens, margin = list(prompt), math.inf
    for _ in range(new_tokens):
        logits = forward(config, weights, tokens)[0][-1].double()
        top = logits.topk(2).values
        margin = min(margin, float((top[0] - top[1]) / logits.std()))
        tokens.append(int(logits.argmax()))
    return tokens[len(prompt):], margin

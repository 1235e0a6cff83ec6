"""Plain, slow restatement of the Tidelorn decoder.  TEST INFRASTRUCTURE ONLY.

One function per mechanism, straight from the equations, on dense tensors of one sequence: no pages, no cache,
no batching and nothing shared with the product path.  Everything is computed in the dtype of ``weights``
(float64 by default: ``random_weights`` draws bf16-representable values and widens them).  ``config`` is the
parsed config.json: ``vocab``, ``width``, ``norm.eps``, ``postln_alpha``, ``embedding``, ``layers``.

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
    """RMS norm whose stored weight is the deviation from one."""

    return unit_rms(x, eps) * (1.0 + weight)


def bigram_rows(tokens: list[int], buckets: int, mul_prev: int, mul_cur: int) -> list[int]:
    """Row of the bigram table for every token of a sequence; the first token takes the extra last row."""

    rows = [buckets]
    for prev, cur in zip(tokens, tokens[1:]):
        rows.append((prev * mul_prev + cur * mul_cur) % buckets)
    return rows[:len(tokens)]


def sinusoid(positions: torch.Tensor, width: int, dtype=torch.float64) -> torch.Tensor:
    """[T, width]: even entries sin, odd entries cos of p * 10000^(-2i / width)."""

    out = torch.zeros(positions.numel(), width, dtype=torch.float64)
    for entry in range(width):
        i = entry // 2
        angle = positions.to(torch.float64) * 10000.0 ** (-2.0 * i / width)
        out[:, entry] = torch.sin(angle) if entry % 2 == 0 else torch.cos(angle)
    return out.to(dtype)


def query_temperature(positions: torch.Tensor, coef: float, every: int, dtype=torch.float64) -> torch.Tensor:
    """[T]: 1 + coef * ln(floor((p + 1) / every) + 1)."""

    blocks = torch.div(positions + 1, every, rounding_mode="floor").to(torch.float64)
    return (1.0 + coef * torch.log(blocks + 1.0)).to(dtype)


def visible(q_pos: int, k_pos: int, window: int | None) -> bool:
    """Causal, and inside the last ``window`` tokens (the token itself included) when there is a window."""

    return 0 <= q_pos - k_pos and (window is None or q_pos - k_pos < window)


def visibility(length: int, window: int | None) -> torch.Tensor:
    """[T, T] boolean matrix of ``visible``."""

    distance = torch.arange(length).unsqueeze(1) - torch.arange(length).unsqueeze(0)
    seen = distance >= 0
    return seen if window is None else seen & (distance < window)


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum_j exp(s_j)) along the last dimension; ``sink`` broadcasts over rows."""

    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink)
    weights = torch.exp(scores - top)
    return weights / (torch.exp(sink - top) + weights.sum(dim=-1, keepdim=True))


def mix_values(v: torch.Tensor, first: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    """Blend of a layer's values with the first value-mixing layer's values of the same token."""

    return (1.0 - lam) * v + lam * first


def clamped_gate(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """g sigmoid(1.702 g) (u + 1) with g clamped from above and u from both sides."""

    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


# -- the model ----------------------------------------------------------------------------------------

def embed(config: dict, weights: dict, tokens: list[int]) -> torch.Tensor:
    table, emb = weights["embed"], config["embedding"]
    big = emb["bigram"]
    x = table[torch.tensor(tokens)] * emb["scale"]
    x = x + weights["bigram"][torch.tensor(bigram_rows(tokens, big["buckets"], big["mul_prev"], big["mul_cur"]))]
    return x + sinusoid(torch.arange(len(tokens)), config["width"], x.dtype)


def attention(config: dict, weights: dict, index: int, h: torch.Tensor, first_values):
    """Output of layer ``index``'s mixer for its input h, and the values the layer projected (before mixing)."""

    layer = config["layers"][index]
    mixer, prefix = layer["mixer"], f"l{index}.mix."
    heads, kv_heads, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    length, eps = h.shape[0], config["norm"]["eps"]
    biased = layer["type"] == "attention"

    def project(name, count, size):
        y = h @ weights[prefix + name].t()
        if biased:
            y = y + weights[prefix + name + ".b"]
        return y.view(length, count, size)

    q, k, v = project("q", heads, dim), project("k", kv_heads, dim), project("v", kv_heads, vdim)
    own = v
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    if layer["type"] == "attention":
        temp = mixer["q_temp"]
        q = q * query_temperature(torch.arange(length), temp["coef"], temp["every"], q.dtype).view(length, 1, 1)
        sinks, window = weights[prefix + "sink"], None
    else:
        sinks, window = torch.zeros(heads, dtype=h.dtype), mixer["mask"]["size"]
    if mixer.get("v_mix") and first_values is not None:
        v = mix_values(v, first_values, weights[prefix + "vmix"])
    seen = visibility(length, window)
    out = torch.empty(length, heads, vdim, dtype=h.dtype)
    for head in range(heads):
        g = head // (heads // kv_heads)
        scores = (q[:, head] @ k[:, g].t()) * mixer["scale"]
        scores = scores.masked_fill(~seen, -math.inf)
        out[:, head] = sink_softmax(scores, sinks[head]) @ v[:, g]
    return out.reshape(length, heads * vdim) @ weights[prefix + "o"].t(), own


def feed_forward(config: dict, weights: dict, index: int, h: torch.Tensor) -> torch.Tensor:
    prefix = f"l{index}.mlp."
    y = clamped_gate(h @ weights[prefix + "gate"].t(), h @ weights[prefix + "up"].t(),
                     config["layers"][index]["mlp"]["limit"])
    return y @ weights[prefix + "down"].t()


def forward(config: dict, weights: dict, tokens: list[int]):
    """``(logits [T, vocab], residual stream after every layer [layers, T, width])`` of one whole sequence."""

    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x = embed(config, weights, tokens)
    streams, first_values = [], None
    for index, layer in enumerate(config["layers"]):
        mixed, own = attention(config, weights, index, x, first_values)
        if layer["mixer"].get("v_mix") and first_values is None:
            first_values = own
        x = rms_norm(alpha * x + mixed, weights[f"l{index}.norm1"], eps)
        if layer["mlp"] is not None:
            x = rms_norm(alpha * x + feed_forward(config, weights, index, x), weights[f"l{index}.norm2"], eps)
        streams.append(x)
    logits = rms_norm(x, weights["final.norm"], eps) @ weights["head"].t()
    return logits, torch.stack(streams)


def greedy(config: dict, weights: dict, prompt: list[int], new_tokens: int):
    """Greedy continuation by recomputing the whole sequence for every token.  Returns ``(tokens, margin)``:
    the smallest top-2 logit gap over the steps divided by the spread of that step's logits."""

    tokens, margin = list(prompt), math.inf
    for _ in range(new_tokens):
        logits = forward(config, weights, tokens)[0][-1].double()
        top = logits.topk(2).values
        margin = min(margin, float((top[0] - top[1]) / logits.std()))
        tokens.append(int(logits.argmax()))
    return tokens[len(prompt):], margin

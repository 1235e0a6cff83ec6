"""Small Tidelorn models for the tests: configurations, bf16-representable random weights, and the same weights as
the oracle's dictionary and as the runner's ``TidelornWeights``."""

from __future__ import annotations

import torch

from mini_inference_engine_b200.engine.model_runner.tidelorn import TidelornShape, TidelornWeights


def full_layer(heads, kv_heads, dim, vdim, *, scale, coef=0.4, every=7, v_mix=True, ff=None, limit=1.5):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "q_temp": {"coef": coef, "every": every}, "v_mix": v_mix},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def window_layer(heads, kv_heads, dim, vdim, window, *, scale, v_mix=True, ff=None, limit=1.5):
    return {"type": "attention_2",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "mask": {"size": window}, "v_mix": v_mix},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def make_config(vocab, width, layers, *, buckets=61, mul_prev=13, mul_cur=5, scale=4.0, eps=1e-5, alpha=1.7):
    return {"architecture": "Tidelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": layers}


# Scores have a standard deviation of about scale * sqrt(dim): around 2, so that single keys stand out.
CONFIGS = {
    # grouped heads, a window first, a mixer without a feed-forward, values mixed from the second layer on
    "grouped": make_config(97, 64, [
        window_layer(4, 2, 16, 24, 5, scale=0.5, v_mix=False, ff=48),
        full_layer(6, 2, 16, 24, scale=0.6, ff=40),
        full_layer(4, 2, 32, 24, scale=0.4, coef=0.25, every=3, ff=None),
        window_layer(8, 2, 24, 24, 20, scale=0.45, ff=56, limit=0.5)]),
    # one key/value head, wide values, alpha and multipliers that are one, a window of one page
    "single_kv": make_config(131, 80, [
        full_layer(10, 1, 40, 72, scale=0.35, coef=0.9, every=16, ff=96, limit=3.0),
        window_layer(10, 1, 40, 72, 16, scale=0.35, ff=32),
        window_layer(3, 1, 8, 72, 33, scale=0.8, v_mix=True, ff=None)],
        buckets=1, mul_prev=1, mul_cur=1, alpha=1.0, scale=1.0),
    # separate heads, no value mixing anywhere, a window of one token
    "separate": make_config(64, 128, [
        full_layer(4, 4, 72, 48, scale=0.25, every=1, v_mix=False, ff=64),
        window_layer(4, 4, 136, 64, 1, scale=0.2, v_mix=False, ff=64),
        window_layer(4, 4, 64, 128, 47, scale=0.3, v_mix=False, ff=64)], buckets=509, mul_prev=31337, mul_cur=7919),
    # sizes no vector width divides: the row kernel and the element-wise glue, no fused head
    "odd": make_config(83, 37, [
        full_layer(3, 1, 10, 7, scale=0.7, ff=23),
        window_layer(6, 1, 5, 7, 9, scale=0.9, ff=11),
        full_layer(2, 1, 3, 7, scale=1.1, coef=0.0, every=1000, ff=None)], eps=1e-3),
}


def make_weights(config: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    """bf16 tensors by checkpoint name, drawn so that every part of a layer matters."""

    generator = torch.Generator().manual_seed(seed)
    out = {}
    for name, size in TidelornShape.from_config(config).tensor_shapes().items():
        noise = torch.randn(size, generator=generator)
        if name == "embed":
            noise = noise / config["embedding"]["scale"]
        elif name.endswith("vmix"):
            noise = torch.rand((), generator=generator) * 0.6 + 0.2
        elif "norm" in name:
            noise = noise * 0.3
        elif name.endswith("sink"):
            noise = noise * 1.5 + 1.0
        elif name.endswith(".b"):
            noise = noise * 0.7
        elif name not in ("bigram",):
            noise = noise * (1.5 / size[1] ** 0.5)
        out[name] = noise.to(torch.bfloat16)
    return out


def oracle_weights(tensors: dict[str, torch.Tensor], dtype=torch.float64) -> dict[str, torch.Tensor]:
    return {name: tensor.to(dtype) for name, tensor in tensors.items()}


def runner_weights(config: dict, tensors: dict[str, torch.Tensor], device, dtype, page: int = 16) -> TidelornWeights:
    return TidelornWeights(TidelornShape.from_config(config, page=page), lambda name, size: tensors[name], device,
                           dtype)


def make_tokens(config: dict, count: int, seed: int) -> list[int]:
    return torch.randint(0, config["vocab"], (count,), generator=torch.Generator().manual_seed(seed)).tolist()


def logit_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Error of every row: root mean square of the centred difference over the vocabulary, in units of the spread
    of the expected logits."""

    difference = got.double().cpu() - want.double()
    difference = difference - difference.mean(dim=-1, keepdim=True)
    return difference.square().mean(dim=-1).sqrt() / want.double().std()


def logit_error(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest row error."""

    return float(logit_errors(got, want).max())

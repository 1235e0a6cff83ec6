"""Small Ripesun models for the tests: configurations, bf16-representable random weights, and the same weights as the
oracle's dictionary and as the runner's ``RipesunWeights``."""

from __future__ import annotations

import torch

from mini_inference_engine_b200.engine.model_runner.ripesun import RipesunShape, RipesunWeights


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, *, scale, base=1e4, rotated=None, kv_from=None, ff=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "mask": {"size": window}, "scale": scale, "rot": {"base": base, "dims": rot_dim if rotated is None else rotated}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def lightning_layer(dim, vdim, decay, *, ff=None):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mingru_layer(size, *, ff=None):
    return {"type": "mingru", "mixer": {"width": size}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def make_config(vocab, width, layers, *, side=8, eps=1e-5, mult=0.7, scale=2.5, cap=9.0):
    return {"architecture": "Ripesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale}, "token_side": {"dim": side}, "logit_softcap": cap, "layers": layers}


# Scores have a standard deviation of about scale * sqrt(dim + rot_dim): around 2, so that single keys stand out.
CONFIGS = {
    # a recurrent layer first; two cached layers, each read by a later one with other heads, sizes and window
    "mixed": make_config(97, 72, [
        lightning_layer(24, 40, (0.5, 0.97, 0.8), ff=56),
        latent_layer(4, 16, 8, 24, 32, 40, 20, scale=0.45, ff=48),
        mingru_layer(48, ff=40),
        latent_layer(6, 24, 16, 16, 24, 56, 7, scale=0.35, base=500.0, ff=None),
        latent_layer(3, 8, 8, 40, 16, 40, 45, scale=0.55, kv_from=1, ff=64),
        latent_layer(5, 32, 16, 8, 40, 56, 16, scale=0.3, base=500.0, kv_from=3, ff=32)]),
    # more than 16 heads, a partly rotated key part, two 64-dim groups of keys and values in the recurrence, a window of
    # one token, no feed-forward after the recurrent layers, factors that are one
    "wide": make_config(131, 96, [
        latent_layer(20, 40, 24, 16, 48, 136, 33, scale=0.3, rotated=16, ff=80),
        lightning_layer(72, 72, (0.9,), ff=None),
        latent_layer(18, 16, 24, 24, 64, 136, 1, scale=0.4, rotated=16, kv_from=0, ff=64),
        mingru_layer(200, ff=None)], side=16, mult=1.0, scale=1.0, cap=20.0, eps=1e-3),
    # a latent of eight 64-dim groups and a key part of one, as large models have it; 40 heads in two groups
    "deep_latent": make_config(80, 64, [
        latent_layer(40, 16, 64, 8, 32, 512, 100, scale=0.2, base=1e6, ff=48),
        lightning_layer(128, 64, (0.99, 0.3), ff=48),
        latent_layer(16, 32, 64, 128, 32, 512, 60, scale=0.2, base=1e6, kv_from=0, ff=48)], side=40, cap=6.0),
    # sizes no vector width divides: the row kernels, the token-by-token recurrence, no fused head
    "odd": make_config(83, 37, [
        latent_layer(3, 5, 6, 7, 9, 11, 9, scale=0.6, rotated=4, ff=23),
        lightning_layer(5, 7, (0.95, 0.6, 1.0), ff=11),
        mingru_layer(13, ff=None),
        latent_layer(1, 10, 6, 3, 5, 11, 30, scale=0.5, rotated=4, kv_from=0, ff=19)], side=11, mult=0.4, scale=3.5),
}


def make_weights(config: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    """bf16 tensors by checkpoint name, drawn so that every part of a layer matters."""

    generator = torch.Generator().manual_seed(seed)
    out = {}
    for name, size in RipesunShape.from_config(config).tensor_shapes().items():
        noise = torch.randn(size, generator=generator)
        if name == "embed":
            noise = noise / config["embedding"]["scale"]
        elif "norm" in name:
            noise = noise * 0.3 + 1.0
        elif name.endswith("sink"):
            noise = noise * 1.5 + 1.0
        elif name.endswith(".b"):
            noise = noise * 0.7
        elif name != "side.embed":
            noise = noise * (1.5 / size[1] ** 0.5)
        out[name] = noise.to(torch.bfloat16)
    return out


def oracle_weights(tensors: dict[str, torch.Tensor], dtype=torch.float64) -> dict[str, torch.Tensor]:
    return {name: tensor.to(dtype) for name, tensor in tensors.items()}


def runner_weights(config: dict, tensors: dict[str, torch.Tensor], device, dtype, page: int = 16) -> RipesunWeights:
    return RipesunWeights(RipesunShape.from_config(config, page=page), lambda name, size: tensors[name], device, dtype)


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

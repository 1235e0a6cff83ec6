"""Model designs this package serves, chosen by ``config.json``.

A design brings its configuration parser, its weights and its runner (a ``PagedStepRunner``); everything around
them - pages, graphs, continuous batching, greedy sampling, the command line - is shared.  ``config.json`` names
its design in ``architecture`` or, as Hugging Face writes it, in ``architectures``.
"""

from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path
from typing import Callable

import torch

from .checkpoint import Checkpoint, CheckpointError, load_config
from .model_runner.qwen3_decode import Qwen3DecodeRunner, Qwen3Shape, Qwen3Weights
from .model_runner.ripesun import RipesunRunner, RipesunShape, RipesunWeights
from .model_runner.step_runner import PagedStepRunner
from .model_runner.tidelorn import TidelornRunner, TidelornShape, TidelornWeights

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class UnsupportedDtype(ValueError):
    """The design does not run in the number format that was asked for."""


@dataclass(frozen=True)
class ModelDesign:
    name: str
    dtypes: tuple[torch.dtype, ...]
    shape: Callable[[dict], object]                  # config -> shape
    checkpoint_weights: Callable                     # (shape, Checkpoint, device, dtype) -> weights
    random_weights: Callable                         # (shape, device, dtype, seed) -> weights
    runner: Callable[..., PagedStepRunner]           # (weights, num_pages=, max_batch=, max_context=, ...) -> runner
    recurrent: bool = False                          # requests hold a state slot; the runner takes state_slots=


DESIGNS: dict[str, ModelDesign] = {}


def register(design: ModelDesign, *aliases: str) -> ModelDesign:
    for name in (design.name, *aliases):
        if name in DESIGNS:
            raise ValueError(f"a design named {name!r} is registered already")
        DESIGNS[name] = design
    return design


def design_for(config: dict) -> ModelDesign:
    names = [config["architecture"]] if "architecture" in config else list(config.get("architectures") or [])
    for name in names:
        if name in DESIGNS:
            return DESIGNS[name]
    raise CheckpointError(f"no registered design for {names or 'a config without an architecture'}; "
                          f"known: {sorted(DESIGNS)}")


def load_runner(folder: str | Path, *, dtype: torch.dtype = torch.bfloat16, device: torch.device | None = None,
                random_seed: int | None = None, state_slots: int | None = None, **runner_options) -> PagedStepRunner:
    """Runner of the model in ``folder``: its checkpoint's weights, or seeded random ones of its configuration
    when ``random_seed`` is given.  ``state_slots`` goes to designs with recurrent state, ``runner_options``
    (``num_pages``, ``max_batch``, ``max_context`` and so on) to every runner."""

    config = load_config(folder)
    design = design_for(config)
    if dtype not in design.dtypes:
        raise UnsupportedDtype(f"{design.name} does not run in {dtype}")
    device = device if device is not None else torch.device("cuda", torch.cuda.current_device())
    shape = design.shape(config)
    if random_seed is None:
        weights = design.checkpoint_weights(shape, Checkpoint(folder), device, dtype)
    else:
        weights = design.random_weights(shape, device, dtype, random_seed)
    if design.recurrent and state_slots is not None:
        runner_options["state_slots"] = state_slots
    return design.runner(weights, **runner_options)


def _qwen3_shape(config: dict) -> Qwen3Shape:
    default = Qwen3Shape()
    rope = config.get("rope_parameters") or {}
    return Qwen3Shape(
        layers=int(config["num_hidden_layers"]), hidden=int(config["hidden_size"]),
        q_heads=int(config["num_attention_heads"]), kv_heads=int(config["num_key_value_heads"]),
        head_dim=int(config.get("head_dim", default.head_dim)), intermediate=int(config["intermediate_size"]),
        vocab=int(config["vocab_size"]), rms_eps=float(config.get("rms_norm_eps", default.rms_eps)),
        rope_theta=float(config.get("rope_theta", rope.get("rope_theta", default.rope_theta))))


def _qwen3_checkpoint(shape, checkpoint, device, dtype):
    raise CheckpointError("the Qwen3 runner has no checkpoint loader: it runs seeded random weights")


register(ModelDesign(
    name="Qwen3ForCausalLM", dtypes=(torch.bfloat16,), shape=_qwen3_shape, checkpoint_weights=_qwen3_checkpoint,
    random_weights=lambda shape, device, dtype, seed: Qwen3Weights(shape, device, seed=seed),
    runner=Qwen3DecodeRunner), "Qwen3")

register(ModelDesign(
    name="Tidelorn", dtypes=(torch.bfloat16, torch.float32), shape=TidelornShape.from_config,
    checkpoint_weights=lambda shape, checkpoint, device, dtype: TidelornWeights(shape, checkpoint.take, device, dtype),
    random_weights=lambda shape, device, dtype, seed: TidelornWeights.random(shape, device, seed=seed, dtype=dtype),
    runner=TidelornRunner))

register(ModelDesign(
    name="Ripesun", dtypes=(torch.bfloat16, torch.float32), shape=RipesunShape.from_config,
    checkpoint_weights=lambda shape, checkpoint, device, dtype: RipesunWeights(shape, checkpoint.take, device, dtype),
    random_weights=lambda shape, device, dtype, seed: RipesunWeights.random(shape, device, seed=seed, dtype=dtype),
    runner=RipesunRunner, recurrent=True))


__all__ = ["DESIGNS", "DTYPES", "ModelDesign", "UnsupportedDtype", "design_for", "load_runner", "register"]

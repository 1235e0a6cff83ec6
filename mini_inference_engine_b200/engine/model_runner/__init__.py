"""Flat-token model loops of the hot path."""

from .qwen3_decode import Qwen3DecodeRunner, Qwen3Shape, Qwen3Weights
from .step_runner import DecodeBuffers, PagedStepRunner

__all__ = ["DecodeBuffers", "PagedStepRunner", "Qwen3DecodeRunner", "Qwen3Shape", "Qwen3Weights"]

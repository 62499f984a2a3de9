"""The model registry: which configuration, weight loading and decoder a model folder's config.json asks for.

An Architecture turns (config, tensors) into a StepDecoder; everything that runs models (the command line, the trace runner,
serving.NativeDecoder) works on that, so a new model is one entry here plus the parts it does not share."""

from collections.abc import Callable
from dataclasses import dataclass
from pathlib import Path

import torch

from .checkpoint import read_config, read_folder
from .decoder import Decoder, DecoderConfig, DecoderWeights, StepDecoder
from .hybrid import HybridConfig, HybridDecoder, HybridWeights
from .native import build_libraries


@dataclass(frozen=True)
class Architecture:
    """build(config, tensors, n_slots, max_len, dtype, device, **decoder options); dtypes it runs in and, by dtype, the
    native libraries it needs (built together before the first launch)."""
    build: Callable[..., StepDecoder]
    libraries: dict[torch.dtype, tuple[str, ...]]

    @property
    def dtypes(self) -> tuple[torch.dtype, ...]:
        return tuple(self.libraries)


ARCHITECTURES: dict[str, Architecture] = {}


def register(*names: str, libraries: dict[torch.dtype, tuple[str, ...]]):
    def add(build: Callable[..., StepDecoder]) -> Callable[..., StepDecoder]:
        for name in names:
            ARCHITECTURES[name] = Architecture(build, libraries)
        return build
    return add


@register("Pudisun", libraries={torch.bfloat16: ("decode_step", "stream_gemm", "tile_gemm", "latent_attn", "gla"),
                                torch.float32: ("decode_step", "gemm_f32", "latent_attn", "gla")})
def build_pudisun(config: dict, tensors: dict, n_slots: int, max_len: int, dtype: torch.dtype, device, **options):
    cfg = HybridConfig.from_pudisun(config, max_len)
    cfg.itemsize = dtype.itemsize
    return HybridDecoder(cfg, HybridWeights.from_state_dict(tensors, cfg, dtype, device), n_slots, device, **options)


@register("Rekudra", libraries={torch.bfloat16: ("decode_step", "stream_gemm", "tile_gemm", "short_conv", "gqa_attn", "delta_rule"),
                                torch.float32: ("decode_step", "gemm_f32", "short_conv", "gqa_attn", "delta_rule")})
def build_rekudra(config: dict, tensors: dict, n_slots: int, max_len: int, dtype: torch.dtype, device, **options):
    cfg = HybridConfig.from_rekudra(config, max_len)
    cfg.itemsize = dtype.itemsize
    return HybridDecoder(cfg, HybridWeights.from_state_dict(tensors, cfg, dtype, device), n_slots, device, **options)


@register("NanochatForCausalLM", "nanochat",
          libraries={torch.bfloat16: ("kv_append", "decode_attn", "decode_step", "stream_gemm", "tile_gemm")})
def build_nanochat(config: dict, tensors: dict, n_slots: int, max_len: int, dtype: torch.dtype, device, **options):
    cfg = DecoderConfig.from_exported(config, max_len)
    return Decoder(cfg, DecoderWeights.from_state_dict(tensors, cfg, device), n_slots, device, **options)


def architecture_of(config: dict) -> Architecture:
    """By "architecture", "architectures" or "model_type", whichever of them names a registered model."""
    names = [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type")]
    for name in names:
        if name in ARCHITECTURES:
            return ARCHITECTURES[name]
    raise ValueError(f"no model for {[n for n in names if n]} (known: {', '.join(sorted(ARCHITECTURES))})")


class UnsupportedDtype(ValueError):
    """The model does not run in the number format asked for."""


def load_decoder(folder: "str | Path", n_slots: int, max_len: int, dtype: torch.dtype = torch.bfloat16,
                 device: "torch.device | str" = "cuda", **options) -> StepDecoder:
    """The decoder of a model folder, weights on the device, with n_slots slots of max_len positions."""
    arch = architecture_of(read_config(folder))
    if dtype not in arch.dtypes:
        raise UnsupportedDtype(f"this model runs in {', '.join(str(d) for d in arch.dtypes)}, not in {dtype}")
    build_libraries(arch.libraries[dtype])
    config, tensors = read_folder(folder)
    return arch.build(config, tensors, n_slots, max_len, dtype, torch.device(device), **options)

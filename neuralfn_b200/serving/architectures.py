"""Model directories by architecture: ``config.json`` names the design, the entry registered for it reads the configuration, says which
native sources its engine needs, and loads the weights (``model.safetensors`` or shards) into a ``ResidentEngine``.

    eng = load_model_directory("/models/some-model", max_batch=8, max_seq=4096)

Hugging Face style configurations name a list (``architectures``), this framework's own designs one name (``architecture``).
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Callable, Mapping

__all__ = ["ArchitectureError", "ModelArchitecture", "ARCHITECTURES", "architecture_of", "is_model_directory", "load_model_directory",
           "read_model_config"]


class ArchitectureError(ValueError):
    pass


@dataclass(frozen=True)
class ModelArchitecture:
    name: str
    family: str                                    # key of native_registry.NATIVE_FAMILIES
    component: str                                 # native library the engine needs (``ops._build.COMPONENTS``)
    dtypes: tuple[str, ...]
    steps: bool                                    # mixed steps (``ResidentEngine.step``)
    build: Callable[..., tuple[Any, dict]]         # (directory, raw config, limits) -> (engine config, engine tensors)


def _build_bulidra(directory: Path, raw: Mapping[str, Any], **limits):
    from ..checkpoint.safetensors_io import read_sharded_checkpoint
    from ..models.bulidra import BulidraConfig, engine_config, pack_tensors
    cfg = BulidraConfig.from_dict(raw)
    return engine_config(cfg, **limits), pack_tensors(cfg, read_sharded_checkpoint(directory))


def _build_murilorn(directory: Path, raw: Mapping[str, Any], **limits):
    from ..checkpoint.safetensors_io import read_sharded_checkpoint
    from ..models.murilorn import MurilornConfig, engine_config, pack_tensors
    tensors = read_sharded_checkpoint(directory)
    cfg = MurilornConfig.from_dict(raw, tensors)
    return engine_config(cfg, **limits), pack_tensors(cfg, tensors)


def _build_vopozen(directory: Path, raw: Mapping[str, Any], **limits):
    from ..checkpoint.safetensors_io import read_sharded_checkpoint
    from ..models.vopozen import VopozenConfig, engine_config, pack_tensors
    tensors = read_sharded_checkpoint(directory)
    cfg = VopozenConfig.from_dict(raw, tensors)
    return engine_config(cfg, **limits), pack_tensors(cfg, tensors)


def _build_kidolorn(directory: Path, raw: Mapping[str, Any], **limits):
    from ..checkpoint.safetensors_io import read_sharded_checkpoint
    from ..models.kidolorn import KidolornConfig, engine_config, pack_tensors
    cfg = KidolornConfig.from_dict(raw)
    return engine_config(cfg, **limits), pack_tensors(cfg, read_sharded_checkpoint(directory))


def _build_hf_llama(directory: Path, raw: Mapping[str, Any], *, max_batch: int = 1, max_seq: int | None = None, dtype: str = "bfloat16", **other):
    from ..checkpoint.safetensors_io import load_hf_llama_directory
    if dtype != "bfloat16":
        raise ArchitectureError("the Llama engine computes in bfloat16")
    if any(v for v in other.values()):
        raise ArchitectureError(f"settings of step engines: {sorted(k for k, v in other.items() if v)}")
    return load_hf_llama_directory(directory, max_batch=max_batch, max_seq=max_seq)


ARCHITECTURES: dict[str, ModelArchitecture] = {a.name: a for a in (
    ModelArchitecture("Bulidra", "bulidra", "layered", ("bfloat16", "float32"), True, _build_bulidra),
    ModelArchitecture("Murilorn", "murilorn", "layered", ("bfloat16", "float32"), True, _build_murilorn),
    ModelArchitecture("Vopozen", "vopozen", "layered", ("bfloat16", "float32"), True, _build_vopozen),
    ModelArchitecture("Kidolorn", "kidolorn", "layered", ("bfloat16", "float32"), True, _build_kidolorn),
    ModelArchitecture("LlamaForCausalLM", "llama", "all", ("bfloat16",), False, _build_hf_llama),
)}


def read_model_config(directory: str | Path) -> dict:
    path = Path(directory) / "config.json"
    if not path.is_file():
        raise ArchitectureError(f"{directory} has no config.json")
    raw = json.loads(path.read_text(encoding="utf-8"))
    if not isinstance(raw, dict):
        raise ArchitectureError(f"{path} must hold a JSON object")
    return raw


def architecture_of(raw: Mapping[str, Any]) -> ModelArchitecture:
    names = [raw["architecture"]] if "architecture" in raw else list(raw.get("architectures") or [])
    for n in names:
        if n in ARCHITECTURES:
            return ARCHITECTURES[n]
    raise ArchitectureError(f"no engine for architecture {names or '(none named)'}; known: {', '.join(sorted(ARCHITECTURES))}")


def is_model_directory(directory: str | Path) -> bool:
    try:
        architecture_of(read_model_config(directory))
        return True
    except (ArchitectureError, ValueError, OSError):
        return False


def load_model_directory(directory: str | Path, *, device: int = 0, **limits):
    """``limits``: ``max_batch``, ``max_seq``, and for step engines ``dtype``, ``kv_tokens``, ``max_step_rows``, ``use_cuda_graph``."""
    from .engine import ResidentEngine
    raw = read_model_config(directory)
    cfg, tensors = architecture_of(raw).build(Path(directory), raw, **limits)
    eng = ResidentEngine(cfg, device=device)
    eng.load_named_tensors(tensors)
    return eng

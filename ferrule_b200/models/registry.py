"""Model registry: which architecture a checkpoint directory holds, and how this build loads and runs it.

An entry names the architecture, recognises its `config.json`, loads its weights, and builds the runner that binds
them to the engine.  `build_runner` is what the command line, the server and the trace runner use.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional

import torch

from ..io.safetensors import CheckpointError


@dataclass(frozen=True)
class RunnerLimits:
    """Sizes a runner is built for."""
    n_pages: int
    page_size: int
    max_rows: int
    max_seqs: int
    max_seq_len: int


@dataclass(frozen=True)
class Architecture:
    name: str
    matches: Callable[[dict], bool]
    load: Callable[..., object]                                  # (directory, device, dtype, max_layers) -> weights
    runner: Callable[..., object]                                # (weights, limits, **options) -> ModelRunner
    dtypes: tuple = (torch.bfloat16,)                            # dtypes its kernel path runs in
    component: str = ""                                          # part of the native library it needs ("": all of it)


def _load_layered(directory, device, dtype, max_layers=0):
    from ..io.layered_checkpoint import load_layered
    return load_layered(directory, device=device, dtype=dtype, max_layers=max_layers)


def _run_layered(weights, lim: RunnerLimits, **options):
    from .layered_runner import LayeredRunner
    return LayeredRunner(weights, n_pages=lim.n_pages, page_size=lim.page_size, max_rows=lim.max_rows, max_seqs=lim.max_seqs,
                         max_seq_len=lim.max_seq_len, **options)


def _load_v4(directory, device, dtype, max_layers=0):
    from ..io.v4_checkpoint import load_v4_hf
    return load_v4_hf(directory, device=device, max_layers=max_layers)


def _run_v4(weights, lim: RunnerLimits, **options):
    from .v4_runner import V4Runner
    return V4Runner(weights, n_pages=lim.n_pages, page_size=lim.page_size, max_seqs=lim.max_seqs,
                    max_seq_len=lim.max_seq_len, max_rows=lim.max_rows, **options)


def _load_deepseek(directory, device, dtype, max_layers=0):
    from ..io.checkpoint import load_deepseek_hf
    return load_deepseek_hf(directory, device=device, dtype=dtype, max_layers=max_layers)


def _run_deepseek(weights, lim: RunnerLimits, **options):
    from .runner import DeepSeekRunner
    return DeepSeekRunner(weights, n_pages=lim.n_pages, page_size=lim.page_size, max_rows=lim.max_rows,
                          max_seqs=lim.max_seqs, max_seq_len=lim.max_seq_len, **options)


ARCHITECTURES: Dict[str, Architecture] = {a.name: a for a in (
    Architecture("gitozen", lambda c: c.get("architecture") == "Gitozen", _load_layered, _run_layered,
                 (torch.bfloat16, torch.float32), "layered"),
    Architecture("supisun", lambda c: c.get("architecture") == "Supisun", _load_layered, _run_layered,
                 (torch.bfloat16, torch.float32), "layered"),
    Architecture("vedadra", lambda c: c.get("architecture") == "Vedadra", _load_layered, _run_layered,
                 (torch.bfloat16, torch.float32), "layered"),
    Architecture("vogunex", lambda c: c.get("architecture") == "Vogunex", _load_layered, _run_layered,
                 (torch.bfloat16, torch.float32), "layered"),
    Architecture("deepseek_v4", lambda c: c.get("model_type") == "deepseek_v4", _load_v4, _run_v4),
    # every other HuggingFace-style config.json is read as a DeepSeek-V2 / V3 model, whose loader checks it
    Architecture("deepseek", lambda c: "architecture" not in c, _load_deepseek, _run_deepseek),
)}


def read_config(directory: str) -> Optional[dict]:
    try:
        with open(os.path.join(directory, "config.json")) as f:
            c = json.load(f)
    except OSError:
        return None
    except ValueError as exc:
        raise CheckpointError(f"{directory}: config.json is not JSON") from exc
    if not isinstance(c, dict):
        raise CheckpointError(f"{directory}: config.json is not a JSON object")
    return c


def architecture_of(directory: str) -> Architecture:
    """The registry entry for a checkpoint directory (by its config.json)."""
    c = read_config(directory)
    if c is None:
        return ARCHITECTURES["deepseek"]             # its loader reports what is missing
    for a in ARCHITECTURES.values():
        if a.matches(c):
            return a
    raise CheckpointError(f"{directory}: unknown architecture {c.get('architecture')!r} "
                          f"(known: {', '.join(sorted(ARCHITECTURES))})")

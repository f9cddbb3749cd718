"""Checkpoint directories of layer-list models (Gitozen, Supisun, Vedadra, Vogunex): `config.json` with one entry per layer, and safetensors
files whose tensors are named `embed`, `pos`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.rg1`, `final.norm`, `head`
(`LayeredConfig.tensor_shapes` lists them).  Linear weights are stored [out, in] in BF16."""
from __future__ import annotations

import json
from dataclasses import replace
from pathlib import Path

import torch

from ..models.layered_config import DeltaMixer, LayeredConfig, from_layer_list, to_layer_list
from ..models.layered_weights import LayeredWeights, RandomTensors, pack_weights
from .safetensors import CheckpointError, ShardedCheckpoint, fails_closed, write_sharded


def bind_config(cfg: LayeredConfig, ck: ShardedCheckpoint) -> LayeredConfig:
    """The sizes only the tensors know: the inner widths of the delta mixers' low-rank projections."""
    layers = list(cfg.layers)
    for i in cfg.delta_layers:
        m = layers[i].mixer
        assert isinstance(m, DeltaMixer)
        if not m.low_rank:
            continue
        ranks = {}
        for field, tensor in (("decay_rank", "a1"), ("gate_rank", "g1")):
            name = f"l{i}.mix.{tensor}"
            if not ck.has(name):
                raise CheckpointError(f"tensor {name} is not in the checkpoint")
            ranks[field] = ck.info(name).shape[0]
        layers[i] = replace(layers[i], mixer=replace(m, **ranks))
    return cfg.with_(layers=tuple(layers))


@fails_closed
def load_layered(directory, device="cpu", dtype=torch.bfloat16, max_layers: int = 0) -> LayeredWeights:
    ck = ShardedCheckpoint(directory)
    cfg = from_layer_list(directory)
    if max_layers:
        cfg = cfg.first_layers(max_layers)
    cfg = bind_config(cfg, ck)
    for name, shape in cfg.tensor_shapes().items():
        if not ck.has(name):
            raise CheckpointError(f"tensor {name} is not in the checkpoint")
        got = tuple(ck.info(name).shape)
        if got != tuple(shape) and not (shape == () and got == (1,)):
            raise CheckpointError(f"tensor {name} has shape {list(got)}, the configuration says {list(shape)}")
    weights = pack_weights(cfg, lambda name: ck.read(name).to(device=device, dtype=dtype))
    ck.close()
    return weights


def export_layered(cfg: LayeredConfig, tensors: RandomTensors, directory, shard_bytes: int = 1 << 30) -> None:
    """Write a checkpoint directory from tensors by name (`RandomTensors`, or anything callable with `.names()`)."""
    d = Path(directory)
    d.mkdir(parents=True, exist_ok=True)
    write_sharded({n: tensors(n).to(torch.bfloat16).cpu() for n in tensors.names()}, d, shard_bytes)
    (d / "config.json").write_text(json.dumps(to_layer_list(cfg), indent=1))

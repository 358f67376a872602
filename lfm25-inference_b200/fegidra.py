"""Fegidra: a parallel-block decoder whose layers mix by chunked softmax attention or by a generalised delta rule, with
an input convolution in front of every mixer and PolyNorm feed-forwards.

config.json: `vocab`, `width`, `norm.eps`, `canon.taps`, and `layers`, one entry per layer with `type` ("attention" or
"general_delta"), `mixer` (sizes and constants) and `mlp` ({"kind": "dense", "ff": ...} or null).  Tensors of layer i are
called `l<i>.…`; linear weights are stored [out, in].
"""
from __future__ import annotations

import os
from dataclasses import dataclass

from .checkpoint import Checkpoint
from .stack import AttentionMixer, GeneralDeltaMixer, ParallelLayer, PolyNormFeedForward, StackModel

ARCHITECTURE = "Fegidra"


class ConfigError(ValueError):
    pass


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int
    rot_base: float
    chunk: int


@dataclass(frozen=True)
class GeneralDeltaConfig:
    heads: int
    dim: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: AttentionConfig | GeneralDeltaConfig
    ff: int                      # 0: no feed-forward


@dataclass(frozen=True)
class FegidraConfig:
    vocab: int
    width: int
    norm_eps: float
    taps: int
    layers: tuple[LayerConfig, ...]

    @classmethod
    def from_json(cls, node: dict) -> "FegidraConfig":
        try:
            return cls(int(node["vocab"]), int(node["width"]), float(node["norm"]["eps"]), int(node["canon"]["taps"]),
                       tuple(_layer_config(index, entry) for index, entry in enumerate(node["layers"])))
        except (KeyError, TypeError) as error:
            raise ConfigError(f"malformed {ARCHITECTURE} configuration: {error!r}") from error


def _layer_config(index: int, entry: dict) -> LayerConfig:
    mixer = entry["mixer"]
    if entry["type"] == "attention":
        rot, mask = mixer.get("rot"), mixer.get("mask")
        parsed = AttentionConfig(int(mixer["heads"]), int(mixer["kv_heads"]), int(mixer["dim"]), int(mixer["vdim"]),
                                 float(mixer["scale"]), int(rot["dims"]) if rot else 0,
                                 float(rot["base"]) if rot else 1.0, int(mask["size"]) if mask else 0)
    elif entry["type"] == "general_delta":
        parsed = GeneralDeltaConfig(int(mixer["heads"]), int(mixer["dim"]))
    else:
        raise ConfigError(f"layer {index}: unknown mixer type {entry['type']!r}")
    mlp = entry.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ConfigError(f"layer {index}: unknown feed-forward kind {mlp['kind']!r}")
    return LayerConfig(parsed, int(mlp["ff"]) if mlp is not None else 0)


def _attention(source, prefix: str, config: AttentionConfig, width: int) -> AttentionMixer:
    queries, keys, values = (config.heads * config.dim, config.kv_heads * config.dim, config.kv_heads * config.vdim)
    return AttentionMixer(
        config.heads, config.kv_heads, config.dim, config.vdim, config.scale, config.rot_dims, config.rot_base,
        config.chunk, source(prefix + "q", (queries, width)), source(prefix + "k", (keys, width)),
        source(prefix + "v", (values, width)), source(prefix + "q.b", (queries,)), source(prefix + "k.b", (keys,)),
        source(prefix + "v.b", (values,)), source(prefix + "q.norm", (queries,)), source(prefix + "k.norm", (keys,)),
        source(prefix + "o", (width, config.heads * config.vdim)))


def _general_delta(source, shape, prefix: str, config: GeneralDeltaConfig, width: int) -> GeneralDeltaMixer:
    size = config.heads * config.dim
    rank = shape(prefix + "w1")[0]
    square = (size, width)
    return GeneralDeltaMixer(
        config.heads, config.dim, source(prefix + "r", square), source(prefix + "k", square),
        source(prefix + "v", square), source(prefix + "g", square), source(prefix + "a", square),
        source(prefix + "a.b", (size,)), source(prefix + "w1", (rank, width)), source(prefix + "w2", (size, rank)),
        source(prefix + "w0", (size,)), source(prefix + "norm", (size,)), source(prefix + "o", (width, size)))


def build(config: FegidraConfig, source, shape, device, num_pages: int, num_request_slots: int,
          dtype: str = "bfloat16") -> StackModel:
    """`source(name, shape)` gives a host tensor, `shape(name)` what the checkpoint holds (the decay's rank is a shape)."""
    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        if isinstance(layer.mixer, AttentionConfig):
            mixer = _attention(source, prefix + "mix.", layer.mixer, config.width)
        else:
            mixer = _general_delta(source, shape, prefix + "mix.", layer.mixer, config.width)
        feed_forward = None
        if layer.ff:
            coefficients = tuple(float(value) for value in source(prefix + "mlp.act", (4,)))
            feed_forward = PolyNormFeedForward(source(prefix + "mlp.up", (layer.ff, config.width)),
                                               source(prefix + "mlp.down", (config.width, layer.ff)), coefficients)
        layers.append(ParallelLayer(
            mixer, source(prefix + "norm1", (config.width,)), source(prefix + "canon1", (config.width, config.taps)),
            source(prefix + "norm2", (config.width,)) if layer.ff else None, feed_forward))
    table = (config.vocab, config.width)
    return StackModel(device, layers, source("embed", table), source("head", table),
                      source("final.norm", (config.width,)), config.norm_eps, num_pages, num_request_slots, dtype)


def load(folder: str, config: dict, device, num_pages: int, num_request_slots: int,
         dtype: str = "bfloat16") -> StackModel:
    """The model of a folder that holds config.json (already parsed as `config`) and model.safetensors."""
    checkpoint = Checkpoint(os.path.join(folder, "model.safetensors"))
    return build(FegidraConfig.from_json(config), checkpoint.tensor, checkpoint.shape, device, num_pages,
                 num_request_slots, dtype)


def tensor_shapes(config: FegidraConfig, rank: int) -> dict[str, tuple[int, ...]]:
    """Every tensor of a checkpoint of this configuration, with a decay of `rank`."""
    shapes: dict[str, tuple[int, ...]] = {}

    def note(name, shape):
        shapes[name] = tuple(shape)

    for index, layer in enumerate(config.layers):
        prefix = f"l{index}.mix."
        if isinstance(layer.mixer, AttentionConfig):
            _attention(note, prefix, layer.mixer, config.width)
        else:
            _general_delta(note, lambda name: (rank,), prefix, layer.mixer, config.width)
        prefix = f"l{index}."
        shapes[prefix + "norm1"] = (config.width,)
        shapes[prefix + "canon1"] = (config.width, config.taps)
        if layer.ff:
            shapes[prefix + "norm2"] = (config.width,)
            shapes[prefix + "mlp.up"] = (layer.ff, config.width)
            shapes[prefix + "mlp.down"] = (config.width, layer.ff)
            shapes[prefix + "mlp.act"] = (4,)
    shapes["embed"] = shapes["head"] = (config.vocab, config.width)
    shapes["final.norm"] = (config.width,)
    return shapes


__all__ = ["ARCHITECTURE", "ConfigError", "FegidraConfig", "build", "load", "tensor_shapes"]

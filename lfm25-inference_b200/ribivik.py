"""Ribivik: a decoder whose layers mix by latent attention or by a Mamba-2 recurrence, with a norm before and after every
sublayer, squared-ReLU feed-forwards and capped logits.

config.json: `vocab`, `width`, `norm.eps`, `logit_softcap`, and `layers`, one entry per layer with `type`
("latent_attention" or "mamba2"), `mixer` (sizes and constants) and `mlp` ({"kind": "dense", "ff": ...} or null).  Tensors
of layer i are called `l<i>.…`; linear weights are stored [out, in].
"""
from __future__ import annotations

import os
from dataclasses import dataclass

from .checkpoint import Checkpoint
from .stack import LatentAttentionMixer, SandwichLayer, SquaredReluFeedForward, StackModel, StateSpaceMixer

ARCHITECTURE = "Ribivik"
NORM_SHIFT = 1.0             # norms over the width store their weights as distances from one


class ConfigError(ValueError):
    pass


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_dims: int
    rot_base: float
    kv_from: int | None          # the layer whose latents are read


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Columns that pass the convolution: x | B | C."""
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class LayerConfig:
    mixer: LatentAttentionConfig | Mamba2Config
    ff: int                      # 0: no feed-forward


@dataclass(frozen=True)
class RibivikConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_softcap: float         # 0: logits are not capped
    layers: tuple[LayerConfig, ...]

    @classmethod
    def from_json(cls, node: dict) -> "RibivikConfig":
        try:
            config = cls(int(node["vocab"]), int(node["width"]), float(node["norm"]["eps"]),
                         float(node.get("logit_softcap") or 0.0),
                         tuple(_layer_config(index, entry) for index, entry in enumerate(node["layers"])))
        except (KeyError, TypeError) as error:
            raise ConfigError(f"malformed {ARCHITECTURE} configuration: {error!r}") from error
        _check_sharing(config.layers)
        return config


def _layer_config(index: int, entry: dict) -> LayerConfig:
    mixer = entry["mixer"]
    if entry["type"] == "latent_attention":
        rot = mixer.get("rot")
        owner = mixer.get("kv_from")
        parsed = LatentAttentionConfig(
            int(mixer["heads"]), int(mixer["dim"]), int(mixer["rot_dim"]), int(mixer["vdim"]), int(mixer["q_rank"]),
            int(mixer["kv_rank"]), float(mixer["scale"]), int(rot["dims"]) if rot else 0,
            float(rot["base"]) if rot else 1.0, None if owner is None else int(owner))
    elif entry["type"] == "mamba2":
        parsed = Mamba2Config(int(mixer["heads"]), int(mixer["vdim"]), int(mixer["state"]), int(mixer["groups"]),
                              int(mixer["norm_groups"]), int(mixer["conv"]))
        if parsed.heads % parsed.groups or parsed.inner % parsed.norm_groups:
            raise ConfigError(f"layer {index}: heads and norm do not divide into their groups")
    else:
        raise ConfigError(f"layer {index}: unknown mixer type {entry['type']!r}")
    mlp = entry.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ConfigError(f"layer {index}: unknown feed-forward kind {mlp['kind']!r}")
    return LayerConfig(parsed, int(mlp["ff"]) if mlp is not None else 0)


def _check_sharing(layers: tuple[LayerConfig, ...]) -> None:
    for index, layer in enumerate(layers):
        owner = layer.mixer.kv_from if isinstance(layer.mixer, LatentAttentionConfig) else None
        if owner is None:
            continue
        source = layers[owner].mixer if 0 <= owner < index else None
        if not isinstance(source, LatentAttentionConfig) or source.kv_from is not None:
            raise ConfigError(f"layer {index}: layer {owner} has no latents of its own before it")
        if (source.kv_rank, source.rot_dim) != (layer.mixer.kv_rank, layer.mixer.rot_dim):
            raise ConfigError(f"layer {index}: latents of layer {owner} have other sizes")


def _latent_attention(source, prefix: str, config: LatentAttentionConfig, width: int) -> LatentAttentionMixer:
    owner = config.kv_from is None
    values = config.heads * config.vdim
    return LatentAttentionMixer(
        config.heads, config.dim, config.rot_dim, config.vdim, config.scale, config.rot_dims, config.rot_base,
        source(prefix + "dq", (config.q_rank, width)), source(prefix + "dq.norm", (config.q_rank,)),
        source(prefix + "uq", (config.heads * (config.dim + config.rot_dim), config.q_rank)),
        source(prefix + "dkv", (config.kv_rank + config.rot_dim, width)) if owner else None,
        source(prefix + "dkv.norm", (config.kv_rank,)) if owner else None,
        source(prefix + "uk", (config.heads * config.dim, config.kv_rank)), source(prefix + "uv", (values, config.kv_rank)),
        source(prefix + "g", (values, width)), source(prefix + "o", (width, values)), config.kv_from)


def _mamba2(source, prefix: str, config: Mamba2Config, width: int) -> StateSpaceMixer:
    return StateSpaceMixer(
        config.heads, config.vdim, config.state, config.groups, config.norm_groups,
        source(prefix + "in", (config.inner + config.channels + config.heads, width)),
        source(prefix + "conv", (config.channels, config.taps)), source(prefix + "conv.b", (config.channels,)),
        source(prefix + "dt_bias", (config.heads,)), source(prefix + "A_log", (config.heads,)),
        source(prefix + "D", (config.heads,)), source(prefix + "norm", (config.inner,)),
        source(prefix + "o", (width, config.inner)))


def _layers(config: RibivikConfig, source) -> list[SandwichLayer]:
    layers, vector = [], (config.width,)
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        make = _latent_attention if isinstance(layer.mixer, LatentAttentionConfig) else _mamba2
        mixer = make(source, prefix + "mix.", layer.mixer, config.width)
        norms = [source(prefix + name, vector) for name in ("norm1", "norm1b")]
        if layer.ff:
            norms += [source(prefix + name, vector) for name in ("norm2", "norm2b")]
            feed_forward = SquaredReluFeedForward(source(prefix + "mlp.up", (layer.ff, config.width)),
                                                  source(prefix + "mlp.down", (config.width, layer.ff)))
        else:
            norms += [None, None]
            feed_forward = None
        layers.append(SandwichLayer(mixer, *norms, feed_forward))
    return layers


def build(config: RibivikConfig, source, device, num_pages: int, num_request_slots: int,
          dtype: str = "bfloat16") -> StackModel:
    """`source(name, shape)` gives a host tensor."""
    table = (config.vocab, config.width)
    return StackModel(device, _layers(config, source), source("embed", table), source("head", table),
                      source("final.norm", (config.width,)), config.norm_eps, num_pages, num_request_slots, dtype,
                      NORM_SHIFT, config.logit_softcap)


def load(folder: str, config: dict, device, num_pages: int, num_request_slots: int,
         dtype: str = "bfloat16") -> StackModel:
    """The model of a folder that holds config.json (already parsed as `config`) and model.safetensors."""
    checkpoint = Checkpoint(os.path.join(folder, "model.safetensors"))
    return build(RibivikConfig.from_json(config), checkpoint.tensor, device, num_pages, num_request_slots, dtype)


def tensor_shapes(config: RibivikConfig) -> dict[str, tuple[int, ...]]:
    """Every tensor of a checkpoint of this configuration."""
    shapes: dict[str, tuple[int, ...]] = {}

    def note(name, shape):
        shapes[name] = tuple(shape)

    _layers(config, note)
    shapes["embed"] = shapes["head"] = (config.vocab, config.width)
    shapes["final.norm"] = (config.width,)
    return shapes


__all__ = ["ARCHITECTURE", "ConfigError", "RibivikConfig", "build", "load", "tensor_shapes"]

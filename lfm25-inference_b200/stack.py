"""Layer-stack models: the device tensors behind `lfm25_stack_model` and the executor that steps them.

A design module (for instance `fegidra`) turns a configuration and a checkpoint into a `StackBuilder`'s layers; this
module owns what is common to all of them: packing of projections that share an input, padding to the shapes the
tensor-core GEMMs take, the paged caches, the per-slot records of recurrent state and the C structs.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import numpy as np
import torch

from . import _abi
from ._abi import check, library

PAGE_SIZE = 16
ACTIVATIONS = {"bfloat16": (_abi.ACTIVATION_BF16, torch.bfloat16), "float32": (_abi.ACTIVATION_F32, torch.float32)}
# rows of a weight matrix (output features) per tile of the small-batch tensor-core GEMM, and its K granularity
ROW_MULTIPLE = 128
COLUMN_MULTIPLE = 64


def round_up(value: int, multiple: int) -> int:
    return (value + multiple - 1) // multiple * multiple


@dataclass
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int
    rot_base: float
    chunk: int
    query: torch.Tensor          # [heads * dim, width]
    key: torch.Tensor
    value: torch.Tensor
    query_bias: torch.Tensor | None
    key_bias: torch.Tensor | None
    value_bias: torch.Tensor | None
    query_norm: torch.Tensor
    key_norm: torch.Tensor
    output: torch.Tensor         # [width, heads * vdim]


@dataclass
class GeneralDeltaMixer:
    heads: int
    dim: int
    receptance: torch.Tensor     # r, k, v, gate, removal: [heads * dim, width]
    key: torch.Tensor
    value: torch.Tensor
    gate: torch.Tensor
    removal: torch.Tensor
    removal_bias: torch.Tensor   # [heads * dim]
    decay_down: torch.Tensor     # [rank, width]
    decay_up: torch.Tensor       # [heads * dim, rank]
    decay_base: torch.Tensor     # [heads * dim]
    norm: torch.Tensor           # [heads * dim]
    output: torch.Tensor         # [width, heads * dim]


@dataclass
class LatentAttentionMixer:
    heads: int
    dim: int                     # unrotated query / key size per head
    rot_dim: int                 # rotated part: per head in queries, shared by all heads in keys
    vdim: int
    scale: float
    rot_dims: int                # leading dimensions of the rotated part that turn
    rot_base: float
    query_down: torch.Tensor     # [q_rank, width]
    query_latent_norm: torch.Tensor
    query_up: torch.Tensor       # [heads * (dim + rot_dim), q_rank]
    latent_down: torch.Tensor | None       # [kv_rank + rot_dim, width]; None with cache_of
    latent_norm: torch.Tensor | None       # [kv_rank]
    key_up: torch.Tensor         # [heads * dim, kv_rank]
    value_up: torch.Tensor       # [heads * vdim, kv_rank]
    gate: torch.Tensor           # [heads * vdim, width]
    output: torch.Tensor         # [width, heads * vdim]
    cache_of: int | None         # the layer whose latents this one reads; None: its own


@dataclass
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    projection: torch.Tensor     # z | x | B | C | dt rows of [.., width]
    conv: torch.Tensor           # [channels, taps] over x | B | C
    conv_bias: torch.Tensor
    step_bias: torch.Tensor      # [heads]
    log_rate: torch.Tensor       # [heads]
    skip: torch.Tensor           # [heads]
    norm: torch.Tensor           # [heads * vdim]
    output: torch.Tensor         # [width, heads * vdim]


@dataclass
class PolyNormFeedForward:
    up: torch.Tensor             # [ff, width]
    down: torch.Tensor           # [width, ff]
    coefficients: tuple[float, float, float, float]


@dataclass
class SquaredReluFeedForward:
    up: torch.Tensor             # [ff, width]
    down: torch.Tensor           # [width, ff]


@dataclass
class ParallelLayer:
    """x <- x + (mixer(h + conv(h)) + feed_forward(n)); `feed_forward` None: x <- x + mixer(h + conv(h))."""

    mixer: AttentionMixer | GeneralDeltaMixer
    mixer_norm: torch.Tensor
    conv: torch.Tensor           # [width, taps]
    ff_norm: torch.Tensor | None
    feed_forward: PolyNormFeedForward | None


@dataclass
class SandwichLayer:
    """x <- x + N(mixer(N(x; mixer_norm)); mixer_post_norm), then the same around the feed-forward unless it is None."""

    mixer: LatentAttentionMixer | StateSpaceMixer
    mixer_norm: torch.Tensor
    mixer_post_norm: torch.Tensor
    ff_norm: torch.Tensor | None
    ff_post_norm: torch.Tensor | None
    feed_forward: SquaredReluFeedForward | None


class StackModel:
    """Weights, caches and recurrent state of a layer-stack model, resident on `device`."""

    def __init__(self, device, layers: list[ParallelLayer] | list[SandwichLayer], embedding: torch.Tensor,
                 head: torch.Tensor, final_norm: torch.Tensor, norm_eps: float, num_pages: int, num_request_slots: int,
                 dtype: str = "bfloat16", norm_shift: float = 0.0, logit_softcap: float = 0.0):
        if dtype not in ACTIVATIONS:
            raise ValueError(f"unknown activation type {dtype}")
        activation, self.dtype = ACTIVATIONS[dtype]
        self.device, self.num_pages, self.num_request_slots = device, num_pages, num_request_slots
        self.vocab, self.width = embedding.shape
        self.norm_eps = norm_eps
        self.sandwich = isinstance(layers[0], SandwichLayer)
        self._element = torch.empty(0, dtype=self.dtype).element_size()
        self._kept = []                      # everything the C structs point into
        self._record_bytes = 0
        self.caches = []                     # per layer with a cache of its own: (key cache, value cache)
        self._layer_caches = {}
        array = (_abi.StackLayer * len(layers))()
        for index, layer in enumerate(layers):
            if isinstance(layer, SandwichLayer) != self.sandwich:
                raise ValueError(f"layer {index}: arrangements of both kinds in one model")
            array[index] = (self._sandwich_layer if self.sandwich else self._parallel_layer)(index, layer)
        self._layer_array = array
        self.record_bytes = round_up(max(self._record_bytes, 1), 256)
        self.records = torch.zeros(num_request_slots * self.record_bytes, dtype=torch.uint8, device=device)
        self.struct = _abi.StackModel(
            len(layers), array, activation, _abi.BLOCK_SANDWICH if self.sandwich else _abi.BLOCK_PARALLEL, self.vocab,
            self.width, norm_eps, norm_shift, logit_softcap, self._keep(embedding), self._keep(final_norm), self._linear([head]), self.records.data_ptr(), self.record_bytes,
            num_request_slots, num_pages)

    # ------------------------------------------------------------------------------------ building the structs

    def _keep(self, tensor: torch.Tensor | None):
        if tensor is None:
            return None
        tensor = tensor.to(self.device).contiguous()
        self._kept.append(tensor)
        return tensor.data_ptr()

    def _linear(self, parts: list[torch.Tensor], section: int = 1) -> _abi.StackLinear:
        """The parts stacked along the output dimension, each padded with zero rows to a multiple of `section` and all of
        them for the tensor-core GEMMs."""
        padding = [torch.zeros((-part.shape[0] % section, part.shape[1]), dtype=torch.bfloat16) for part in parts]
        weight = torch.cat([block.to(self.device, torch.bfloat16) for pair in zip(parts, padding) for block in pair], dim=0)
        rows = round_up(weight.shape[0], ROW_MULTIPLE if weight.shape[0] >= ROW_MULTIPLE else 16)
        padded = torch.zeros((rows, weight.shape[1]), dtype=torch.bfloat16, device=self.device)
        padded[:weight.shape[0]] = weight
        return _abi.StackLinear(self._keep(padded), rows, weight.shape[1])

    def _joined(self, mixer_output: torch.Tensor, down: torch.Tensor | None) -> _abi.StackLinear:
        """[W_o | W_down] side by side; columns padded when a feed-forward follows (its kernel clears the padding)."""
        parts = [mixer_output.to(self.device, torch.bfloat16)]
        if down is not None:
            parts.append(down.to(self.device, torch.bfloat16))
        columns = sum(part.shape[1] for part in parts)
        total = round_up(columns, COLUMN_MULTIPLE) if down is not None else columns
        weight = torch.zeros((self.width, total), dtype=torch.bfloat16, device=self.device)
        weight[:, :columns] = torch.cat(parts, dim=1)
        return _abi.StackLinear(self._keep(weight), self.width, total)

    def _reserve(self, count: int) -> int:
        offset = round_up(self._record_bytes, 256)
        self._record_bytes = offset + count
        return offset

    def _convolution(self, struct: _abi.StackLayer, conv: torch.Tensor) -> None:
        """`conv` [channels, taps]"""
        struct.conv = self._keep(conv.to(torch.bfloat16).t())
        struct.conv_taps = conv.shape[1]
        struct.conv_offset = self._reserve((conv.shape[1] - 1) * conv.shape[0] * self._element)

    def _rotation(self, struct: _abi.StackLayer, dims: int, base: float) -> None:
        struct.rot_dims = dims
        if dims:
            exponents = -2.0 * np.arange(dims // 2, dtype=np.float64) / dims
            struct.inv_freq = self._keep(torch.from_numpy((float(base) ** exponents).astype(np.float32)))

    def _new_cache(self, index: int, key_shape: tuple[int, ...], value_shape: tuple[int, ...]):
        caches = tuple(torch.zeros((self.num_pages, *shape), dtype=self.dtype, device=self.device)
                       for shape in (key_shape, value_shape))
        self.caches.append(caches)
        self._layer_caches[index] = caches
        return caches

    def _parallel_layer(self, index: int, layer: ParallelLayer) -> _abi.StackLayer:
        struct, mixer, ff = _abi.StackLayer(), layer.mixer, layer.feed_forward
        if layer.conv.shape[0] != self.width:
            raise ValueError(f"layer {index}: convolution shape {tuple(layer.conv.shape)}")
        struct.mixer_norm = self._keep(layer.mixer_norm)
        self._convolution(struct, layer.conv)
        struct.heads, struct.dim = mixer.heads, mixer.dim
        if isinstance(mixer, AttentionMixer):
            struct.mixer = _abi.MIXER_ATTENTION
            struct.projection = self._linear([mixer.query, mixer.key, mixer.value])
            struct.kv_heads, struct.vdim, struct.chunk, struct.scale = mixer.kv_heads, mixer.vdim, mixer.chunk, mixer.scale
            self._rotation(struct, mixer.rot_dims, mixer.rot_base)
            biases = [mixer.query_bias, mixer.key_bias, mixer.value_bias]
            if any(bias is not None for bias in biases):
                weights = [mixer.query, mixer.key, mixer.value]
                struct.bias = self._keep(torch.cat(
                    [torch.zeros(weight.shape[0], dtype=torch.bfloat16) if bias is None else bias.cpu()
                     for bias, weight in zip(biases, weights)]))
            struct.query_norm, struct.key_norm = self._keep(mixer.query_norm), self._keep(mixer.key_norm)
            caches = self._new_cache(index, (mixer.kv_heads, PAGE_SIZE, mixer.dim),
                                     (mixer.kv_heads, PAGE_SIZE, mixer.vdim))
            struct.key_cache, struct.value_cache = caches[0].data_ptr(), caches[1].data_ptr()
        else:
            struct.mixer = _abi.MIXER_GENERAL_DELTA
            struct.projection = self._linear([mixer.receptance, mixer.key, mixer.value, mixer.gate, mixer.removal,
                                              mixer.decay_down])
            struct.rank = mixer.decay_down.shape[0]
            struct.decay_up, struct.decay_base = self._keep(mixer.decay_up), self._keep(mixer.decay_base)
            struct.removal_bias, struct.head_norm = self._keep(mixer.removal_bias), self._keep(mixer.norm)
            struct.state_offset = self._reserve(mixer.heads * mixer.dim * mixer.dim * 4)
        struct.output = self._joined(mixer.output, None if ff is None else ff.down)
        if ff is not None:
            struct.ff_norm = self._keep(layer.ff_norm)
            struct.ff = ff.up.shape[0]
            struct.up = self._linear([ff.up])
            struct.poly[:] = ff.coefficients
        return struct

    def _sandwich_layer(self, index: int, layer: SandwichLayer) -> _abi.StackLayer:
        struct, mixer, ff = _abi.StackLayer(), layer.mixer, layer.feed_forward
        struct.mixer_norm, struct.mixer_post_norm = self._keep(layer.mixer_norm), self._keep(layer.mixer_post_norm)
        struct.heads, struct.vdim = mixer.heads, mixer.vdim
        if isinstance(mixer, LatentAttentionMixer):
            self._latent_attention(index, struct, mixer)
        else:
            self._state_space(struct, mixer)
        struct.output = self._joined(mixer.output, None)
        if ff is not None:
            struct.ff_norm, struct.ff_post_norm = self._keep(layer.ff_norm), self._keep(layer.ff_post_norm)
            struct.ff = ff.up.shape[0]
            struct.ff_activation = _abi.FEED_FORWARD_SQUARED_RELU
            struct.up = self._linear([ff.up])
            down = torch.zeros((self.width, struct.up.n), dtype=torch.bfloat16, device=self.device)
            down[:, :struct.ff] = ff.down.to(self.device, torch.bfloat16)
            struct.down = _abi.StackLinear(self._keep(down), self.width, struct.up.n)
        return struct

    def _latent_attention(self, index: int, struct: _abi.StackLayer, mixer: LatentAttentionMixer) -> None:
        struct.mixer = _abi.MIXER_LATENT_ATTENTION
        struct.dim, struct.rot_dim, struct.scale = mixer.dim, mixer.rot_dim, mixer.scale
        struct.q_rank, struct.kv_rank = mixer.query_down.shape[0], mixer.key_up.shape[1]
        self._rotation(struct, mixer.rot_dims, mixer.rot_base)
        struct.query_latent_norm = self._keep(mixer.query_latent_norm)
        if mixer.cache_of is None:
            caches = self._new_cache(index, (PAGE_SIZE, mixer.rot_dim), (PAGE_SIZE, struct.kv_rank))
            struct.latent_norm = self._keep(mixer.latent_norm)
            parts = [mixer.query_down, mixer.latent_down, mixer.gate]
        else:
            caches = self._layer_caches.get(mixer.cache_of)
            if caches is None or tuple(cache.shape[2] for cache in caches) != (mixer.rot_dim, struct.kv_rank):
                raise ValueError(f"layer {index}: layer {mixer.cache_of} has no latents of its sizes")
            struct.shared_cache = 1
            parts = [mixer.query_down, mixer.gate]
        struct.key_cache, struct.value_cache = caches[0].data_ptr(), caches[1].data_ptr()
        struct.projection = self._linear(parts, section=8)
        struct.query_up = self._linear([mixer.query_up])
        struct.latent_up = self._linear([mixer.key_up, mixer.value_up])

    def _state_space(self, struct: _abi.StackLayer, mixer: StateSpaceMixer) -> None:
        struct.mixer = _abi.MIXER_STATE_SPACE
        struct.groups, struct.state_size, struct.norm_groups = mixer.groups, mixer.state, mixer.norm_groups
        struct.projection = self._linear([mixer.projection])
        self._convolution(struct, mixer.conv)
        struct.conv_bias, struct.step_bias = self._keep(mixer.conv_bias), self._keep(mixer.step_bias)
        struct.log_rate, struct.skip = self._keep(mixer.log_rate), self._keep(mixer.skip)
        struct.head_norm = self._keep(mixer.norm)
        struct.state_offset = self._reserve(mixer.heads * mixer.state * mixer.vdim * 4)

    # ------------------------------------------------------------------------------------ framework hooks

    def create_engine(self, blaslt_handle, config: _abi.EngineConfig, out) -> int:
        return library().lfm25_engine_create_stack(blaslt_handle, ctypes.byref(self.struct), ctypes.byref(config), out)

    def weight_bytes(self, use_fp8: bool = False) -> int:
        """Bytes of weights one decode step streams."""
        linears = [self.struct.head]
        for layer in self._layer_array:
            linears += [layer.projection, layer.output, layer.up, layer.down, layer.query_up, layer.latent_up]
        return sum(linear.n * linear.k * 2 for linear in linears)


class StackExecutor:
    """Steps of a `StackModel`; same calls as `model.DecodeExecutor` where the C ABI has them."""

    def __init__(self, blaslt, model: StackModel, maximum_tokens: int, maximum_rows: int | None = None):
        self.blaslt, self.model = blaslt, model
        self._handle = ctypes.c_void_p()
        check(library().lfm25_stack_executor_create(blaslt._handle, ctypes.byref(model.struct), maximum_tokens,
                                                    maximum_tokens if maximum_rows is None else maximum_rows,
                                                    ctypes.byref(self._handle)))

    def forward(self, batch, advance: bool = False) -> None:
        self.blaslt.bind_current_stream()
        check(library().lfm25_stack_executor_forward(self._handle, batch.struct, int(advance)))

    def step_graph(self, batch, advance: bool = True) -> None:
        self.blaslt.bind_current_stream()
        check(library().lfm25_stack_executor_step_graph(self._handle, batch.struct, int(advance)))

    def forward_ragged(self, batch, num_output_rows: int | None = None) -> None:
        """`num_output_rows`: entries of batch.output_rows to answer (default: one per segment)."""
        self.blaslt.bind_current_stream()
        rows = batch.num_segments if num_output_rows is None else num_output_rows
        check(library().lfm25_stack_executor_forward_ragged(self._handle, batch.struct, rows))

    def logits(self, rows: int) -> np.ndarray:
        host = np.empty((rows, self.model.vocab), dtype=np.float32)
        check(library().lfm25_stack_executor_read_logits(self._handle, host.ctypes.data, rows))
        return host

    def sampled(self, count: int) -> np.ndarray:
        host = torch.empty(count, dtype=torch.int32).pin_memory()
        check(library().lfm25_stack_executor_download_sampled(self._handle, host.data_ptr(), count))
        torch.cuda.current_stream().synchronize()
        return host.numpy().view(np.uint32).copy()

    def set_depth(self, layers: int) -> None:
        """Run only the first `layers` layers of later steps (0 = all): a test aid."""
        check(library().lfm25_stack_executor_set_depth(self._handle, layers))

    def residual(self, tokens: int) -> np.ndarray:
        """The f32 residual stream behind the last layer that ran, for the last step's first `tokens` tokens."""
        host = np.empty((tokens, self.model.width), dtype=np.float32)
        check(library().lfm25_stack_executor_read_residual(self._handle, host.ctypes.data, tokens))
        return host

    def graph_kernels(self) -> int:
        return int(library().lfm25_stack_executor_graph_kernels(self._handle))

    def graph_captures(self) -> int:
        return int(library().lfm25_stack_executor_graph_captures(self._handle))

    def close(self) -> None:
        if self._handle:
            library().lfm25_stack_executor_destroy(self._handle)
            self._handle = None

"""Throughput of a layer-stack model beside the closest other model at equal size: decode steps and mixed prefill steps with
random weights, and the device time of every kernel of a step against its roofline.

Fegidra (beside the LFM2 model) has LFM2.5-1.2B's shape: width 2048, 16 layers of which the same six are attention (32 query
and 8 key/value heads of 64), delta-rule layers of 32 heads of 64 in place of the gated convolutions, feed-forwards of
12288 (two matrices with as many weights as SwiGLU's three at 8192), vocabulary 65536.  Ribivik (beside Fegidra) has the
same width, layers, feed-forwards and vocabulary, latent attention (32 heads, latents of 512, a rotated part of 64) and
recurrences of 64 heads of 64 with a state of 128.  All run in BF16.
"""
from __future__ import annotations

import re
from dataclasses import dataclass
from typing import Callable

import numpy as np
import torch

from . import fegidra, ops, ribivik, stack, workloads
from . import model as lfm_model

RANK = 64
TAPS = 4


def fegidra_config(width=2048, num_layers=16, attention_layers=lfm_model.ATTENTION_LAYERS, heads=32, kv_heads=8, dim=64,
           delta_heads=32, delta_dim=64, ff=12288, vocab=lfm_model.VOCAB, chunk=8192) -> dict:
    attention = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk},
                 "rot": {"base": 10000.0, "dims": dim}, "scale": dim ** -0.5}
    delta = {"heads": delta_heads, "dim": delta_dim}
    return {"vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "canon": {"taps": TAPS},
            "layers": [{"type": "attention" if index in attention_layers else "general_delta",
                        "mixer": attention if index in attention_layers else delta,
                        "mlp": {"kind": "dense", "ff": ff}} for index in range(num_layers)]}


def ribivik_config(width=2048, num_layers=16, attention_layers=lfm_model.ATTENTION_LAYERS, heads=32, dim=64, rot_dim=64,
                   vdim=64, q_rank=768, kv_rank=512, ssm_heads=64, ssm_vdim=64, state=128, groups=8, ff=12288,
                   vocab=lfm_model.VOCAB) -> dict:
    attention = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                 "rot": {"base": 10000.0, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5}
    recurrence = {"heads": ssm_heads, "vdim": ssm_vdim, "state": state, "groups": groups, "norm_groups": groups,
                  "conv": TAPS}
    return {"vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
            "layers": [{"type": "latent_attention" if index in attention_layers else "mamba2",
                        "mixer": attention if index in attention_layers else recurrence,
                        "mlp": {"kind": "dense", "ff": ff}} for index in range(num_layers)]}


def _random_source(device, seed: int, special: Callable):
    """`special(name, values)`: the values of a tensor that is not an ordinary matrix or vector, or None."""
    generator = torch.Generator(device=device).manual_seed(seed)

    def source(name, shape):
        values = torch.randn(shape, generator=generator, device=device)
        chosen = special(name, values)
        if chosen is None:
            chosen = values * (shape[1] ** -0.5 if len(shape) == 2 else 0.1)
        return chosen.to(torch.bfloat16)
    return source


def fegidra_model(node: dict, seed: int, device, num_pages: int, slots: int) -> stack.StackModel:
    def special(name, values):
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            return 1.0 + 0.1 * values
        return torch.tensor([0.5, 0.3, 0.2, 0.0], device=device) if name.endswith(".act") else None
    return fegidra.build(fegidra.FegidraConfig.from_json(node), _random_source(device, seed, special), lambda name: (RANK,),
                         device, num_pages, slots)


def ribivik_model(node: dict, seed: int, device, num_pages: int, slots: int) -> stack.StackModel:
    def special(name, values):
        if name.endswith(".norm") and name != "final.norm":
            return 1.0 + 0.1 * values
        return values - 3.0 if name.endswith("dt_bias") else None
    return ribivik.build(ribivik.RibivikConfig.from_json(node), _random_source(device, seed, special), device, num_pages,
                         slots)


@dataclass(frozen=True)
class Step:
    """What a step's kernels have to touch: `keys` visible keys summed over the tokens, `contexts` cached tokens summed over
    the segments."""
    tokens: int
    segments: int
    keys: float
    contexts: float

    @property
    def decode(self) -> bool:
        return self.segments == self.tokens


def timed_ms(run, steps: int, warmup: int = 3) -> float:
    for _ in range(max(warmup, 3)):
        run()
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.current_stream().synchronize()
    start.record()
    for _ in range(steps):
        run()
    stop.record()
    torch.cuda.current_stream().synchronize()
    return start.elapsed_time(stop) / steps


def kernel_times(run, steps: int = 4) -> dict:
    """{kernel: (launches per step, microseconds per launch)} of `run`, from CUPTI activity records.  Programmatic
    dependent launch is off meanwhile: with it a record also covers the time a kernel waits for its predecessor."""
    ops.set_option("pdl", 0)
    try:
        return _kernel_times(run, steps)
    finally:
        ops.set_option("pdl", 1)


def _kernel_times(run, steps: int) -> dict:
    for _ in range(3):                  # a changed switch makes captured steps run eagerly once and be captured again
        run()
    torch.cuda.synchronize()
    with torch.profiler.profile(activities=[torch.profiler.ProfilerActivity.CUDA]) as profiler:
        for _ in range(steps):
            run()
        torch.cuda.synchronize()
    totals: dict[str, list[float]] = {}
    for event in profiler.events():
        if event.device_type == torch.autograd.DeviceType.CUDA and "Mem" not in event.name:
            name = re.sub(r"^void |lfm25::|\(anonymous namespace\)::", "", event.name)
            name = re.split(r"[<(]", name)[0]
            name = "cuBLASLt GEMM" if re.search(r"nvjet|cutlass|gemm_|sm100_xmma", name) and "umma" not in name else name
            entry = totals.setdefault(name, [0, 0.0])
            entry[0] += 1
            entry[1] += float(event.device_time)
    return {name: (count / steps, total / count) for name, (count, total) in
            sorted(totals.items(), key=lambda item: -item[1][1])}


FP32_TFLOPS = 75.0           # nominal rate of f32 multiply-adds outside the tensor cores


def _fegidra_work(node: dict, step: Step) -> dict:
    """Algorithmic bytes (activations, caches and state once; cache rows once per token for decode and once per segment
    else) and flops per launch of the stack's own kernels; the recurrence's flops are f32 multiply-adds."""
    width, layers, tokens, segments = node["width"], node["layers"], step.tokens, step.segments
    attention = next(layer["mixer"] for layer in layers if layer["type"] == "attention")
    delta = next(layer["mixer"] for layer in layers if layer["type"] == "general_delta")
    ff = layers[0]["mlp"]["ff"]
    heads, groups, dim, vdim = attention["heads"], attention["kv_heads"], attention["dim"], attention["vdim"]
    projected = heads * dim + groups * (dim + vdim)
    inner = delta["heads"] * delta["dim"]
    state = delta["heads"] * delta["dim"] ** 2 * 4
    return {
        "residual_norm_conv_kernel": [(tokens * width * (4 + 2 + 4 + 2 + 2) + segments * width * (TAPS - 1) * 4, 0.0, 0.0)],
        "poly_norm_kernel": [(tokens * ff * 4, 0.0, 0.0)],
        "projection_norm_rope_kernel": [(tokens * projected * 4, 0.0, 0.0)],
        "attention": [(step.keys * groups * (dim + vdim) * 2 if step.decode else 0.0,
                       2.0 * step.keys * heads * (dim + vdim), 0.0)],
        "delta": [(tokens * (6 * inner + RANK) * 2 + segments * state * 2, 0.0,
                   tokens * delta["heads"] * delta["dim"] ** 2 * 10.0)],
    }


def _ribivik_work(node: dict, step: Step) -> dict:
    """The same; a kernel that runs more than once per layer has an entry for each launch."""
    width, layers, tokens, segments = node["width"], node["layers"], step.tokens, step.segments
    a = next(layer["mixer"] for layer in layers if layer["type"] == "latent_attention")
    m = next(layer["mixer"] for layer in layers if layer["type"] == "mamba2")
    ff = layers[0]["mlp"]["ff"]
    heads, rank, cached = a["heads"], a["kv_rank"], a["kv_rank"] + a["rot_dim"]
    inner = m["heads"] * m["vdim"]
    channels = inner + 2 * m["groups"] * m["state"]
    state = m["heads"] * m["state"] * m["vdim"] * 4
    recurrence = (tokens * (channels + inner + m["heads"]) * 2 + segments * state * 2, 0.0,
                  tokens * m["heads"] * m["state"] * m["vdim"] * 5.0)
    return {
        "residual_post_norm_kernel": [(tokens * width * (4 + 2 + 4 + 2), 0.0, 0.0)],
        "squared_relu_kernel": [(tokens * ff * 4, 0.0, 0.0)],
        "latent_projection_kernel": [(tokens * (a["q_rank"] + cached) * 4, 0.0, 0.0)],
        "rotate_queries_kernel": [(tokens * heads * a["rot_dim"] * 4, 0.0, 0.0)],
        "head_linear_mma_kernel": [(heads * size * rank * 2 + tokens * heads * (rank + size + gate) * 2,
                                    2.0 * tokens * heads * size * rank, 0.0)
                                   for size, gate in ((a["dim"], 0), (a["vdim"], a["vdim"]))],
        "latent_attention_umma_kernel": [(step.keys * cached * 2, 2.0 * step.keys * heads * (cached + rank), 0.0)],
        "gather_context_kernel": [(step.contexts * cached * 4, 0.0, 0.0)],
        "stack_attention_umma_kernel": [(0.0, 2.0 * step.keys * heads * (a["dim"] + a["rot_dim"] + a["vdim"]), 0.0)],
        "channel_conv_kernel": [(tokens * channels * 4 + segments * channels * (TAPS - 1) * 4, 0.0, 0.0)],
        "state_space_decode_kernel": [recurrence],
        "state_space_chunk_kernel": [recurrence],
        "gated_group_norm_kernel": [(tokens * inner * 6, 0.0, 0.0)],
    }


def _lfm2_work(step: Step) -> dict:
    tokens, segments = step.tokens, step.segments
    return {"rms_norm_kernel": [(tokens * 2048 * 8, 0.0, 0.0)],
            "short_conv": [(tokens * 2048 * 8 + segments * 2048 * 8, 0.0, 0.0)],
            "silu_mul": [(tokens * 8192 * 6, 0.0, 0.0)], "qk_norm_rope": [(tokens * 3072 * 4, 0.0, 0.0)],
            "attention": [(step.keys * 8 * 256 if step.decode else 0.0, 4.0 * step.keys * 2048, 0.0)]}


def rooflines(work: dict, times, hbm_gbs, tensor_tflops) -> dict:
    """Per kernel: achieved over the roofline that bounds it."""
    out = {}
    for kernel, (launches, micros) in times.items():
        launched = work.get(kernel) or next((entry for key, entry in work.items() if key in kernel), None)
        if launched is None:
            continue
        ideal = 1e6 * sum(max(size / (hbm_gbs * 1e9), flops / (tensor_tflops * 1e12), scalar / (FP32_TFLOPS * 1e12))
                          for size, flops, scalar in launched) / len(launched)
        out[kernel] = {"us": round(micros, 2), "roofline_us": round(ideal, 2), "frac": round(ideal / micros, 3)}
    return out


def _summary(milliseconds: float, times: dict, work: dict, tokens: int, hbm: float, tensor: float, **more) -> dict:
    return {"ms_per_step": milliseconds, "tok_s": tokens / milliseconds * 1e3,
            "kernels": {name: [count, round(micros, 2)] for name, (count, micros) in times.items()},
            "rooflines": rooflines(work, times, hbm, tensor), **more}


@dataclass(frozen=True)
class Design:
    """A model of the benchmark: its configuration, how to build it and what its kernels have to touch."""
    name: str
    node: dict
    build: Callable
    work: Callable

    @property
    def limit(self) -> int:
        """Longest range of keys that a token sees, 0 = all."""
        masks = [layer["mixer"].get("mask") for layer in self.node["layers"]]
        return next((mask["size"] for mask in masks if mask), 0)

    def step(self, positions, tokens: int, segments: int, contexts: float) -> Step:
        positions = positions.astype(np.float64)
        return Step(tokens, segments, float((positions % self.limit if self.limit else positions).sum() + tokens), contexts)


def fegidra_design(**sizes) -> Design:
    return Design("fegidra", fegidra_config(**sizes), fegidra_model, _fegidra_work)


def ribivik_design(**sizes) -> Design:
    return Design("ribivik", ribivik_config(**sizes), ribivik_model, _ribivik_work)


def _stack_decode(device, blaslt, design: Design, batch, fixed_batch, steps: int, hbm, tensor) -> dict:
    sequences = len(batch.contexts)
    model = design.build(design.node, 7, device, batch.num_pages, sequences)
    executor = stack.StackExecutor(blaslt, model, sequences)
    device_batch = fixed_batch()
    milliseconds = timed_ms(lambda: executor.step_graph(device_batch, advance=False), steps)
    times = kernel_times(lambda: executor.step_graph(device_batch, advance=False))
    positions = batch.positions(0)
    step = design.step(positions, sequences, sequences, float(positions.sum() + sequences))
    out = _summary(milliseconds, times, design.work(design.node, step), sequences, hbm, tensor,
                   launches=executor.graph_kernels(), weight_bytes=model.weight_bytes())
    executor.close()
    return out


def _lfm2_decode(device, blaslt, batch, fixed_batch, steps: int, hbm, tensor) -> dict:
    sequences = len(batch.contexts)
    reference = lfm_model.RandomModel(7, device, batch.num_pages, sequences, fp8_policy=False)
    closest = lfm_model.DecodeExecutor(blaslt, sequences)
    device_batch = fixed_batch()
    milliseconds = timed_ms(lambda: closest.step_graph(reference, device_batch, use_fp8=False, advance=False), steps)
    times = kernel_times(lambda: closest.step_graph(reference, device_batch, use_fp8=False, advance=False))
    step = Step(sequences, sequences, float(batch.positions(0).astype(np.float64).sum() + sequences), 0.0)
    out = _summary(milliseconds, times, _lfm2_work(step), sequences, hbm, tensor, launches=closest.graph_kernels(),
                   weight_bytes=reference.weight_bytes(False))
    closest.close()
    return out


def decode_case(device, sequences: int, contexts, steps: int, design: Design, beside: Design | str | None, hbm: float,
                tensor: float) -> dict:
    """Decode steps replayed from their graphs, of the stack and, on the same batch, of the model `beside` it ("lfm2" or
    another design)."""
    batch = workloads.ragged_decode_batch(1, sequences, contexts[0], contexts[1],
                                          sequences * (contexts[1] // 16 + 8) + 64, 64)
    token_ids = np.random.default_rng(3).integers(0, design.node["vocab"], size=sequences).astype(np.uint32)
    context = int(batch.contexts.max()) + 64
    out = {"sequences": sequences, "contexts": list(contexts)}

    def fixed_batch():
        return lfm_model.DecodeBatch(device, batch.block_tables, batch.request_slots, batch.positions(0), token_ids,
                                     context)

    blaslt = ops.BlasLt()
    blaslt.bind_current_stream()
    out["stack"] = _stack_decode(device, blaslt, design, batch, fixed_batch, steps, hbm, tensor)
    if beside == "lfm2":
        out["lfm2"] = _lfm2_decode(device, blaslt, batch, fixed_batch, steps, hbm, tensor)
    elif beside is not None:
        out[beside.name] = _stack_decode(device, blaslt, beside, batch, fixed_batch, steps, hbm, tensor)
    blaslt.close()
    torch.cuda.empty_cache()
    return out


def _stack_prefill(device, blaslt, design: Design, batch, pages: int, token_ids, steps: int, hbm, tensor) -> dict:
    model = design.build(design.node, 7, device, pages, batch.num_segments)
    executor = stack.StackExecutor(blaslt, model, batch.num_tokens, batch.num_segments)
    device_batch = lfm_model.RaggedBatch(device, batch, token_ids)
    milliseconds = timed_ms(lambda: executor.forward_ragged(device_batch), steps)
    times = kernel_times(lambda: executor.forward_ragged(device_batch))
    step = design.step(batch.positions, batch.num_tokens, batch.num_segments, float((batch.prefixes + batch.chunks).sum()))
    out = _summary(milliseconds, times, design.work(design.node, step), batch.num_tokens, hbm, tensor)
    executor.close()
    return out


def _lfm2_prefill(device, blaslt, batch, pages: int, token_ids, steps: int, hbm, tensor) -> dict:
    reference = lfm_model.RandomModel(7, device, pages, batch.num_segments, fp8_policy=False)
    closest = lfm_model.DecodeExecutor(blaslt, batch.num_tokens, maximum_segments=batch.num_segments)
    device_batch = lfm_model.RaggedBatch(device, batch, token_ids)
    milliseconds = timed_ms(lambda: closest.forward_ragged(reference, device_batch, use_fp8=False), steps)
    times = kernel_times(lambda: closest.forward_ragged(reference, device_batch, use_fp8=False))
    step = Step(batch.num_tokens, batch.num_segments, float((batch.positions.astype(np.float64) + 1).sum()), 0.0)
    out = _summary(milliseconds, times, _lfm2_work(step), batch.num_tokens, hbm, tensor)
    closest.close()
    return out


def prefill_case(device, prefixes, chunk: int, steps: int, design: Design, beside: Design | str | None, hbm: float,
                 tensor: float) -> dict:
    """Mixed steps of `chunk` new tokens behind each of `prefixes` cached ones."""
    pages = sum((prefix + chunk + 15) // 16 for prefix in prefixes)
    batch = workloads.mixed_step_batch(5, prefixes, [chunk] * len(prefixes), pages)
    token_ids = np.random.default_rng(5).integers(0, design.node["vocab"], size=batch.num_tokens).astype(np.uint32)
    out = {"prefixes": list(prefixes), "chunk": chunk}
    if design.limit:
        out["attention_chunk"] = design.limit
    blaslt = ops.BlasLt()
    blaslt.bind_current_stream()
    out["stack"] = _stack_prefill(device, blaslt, design, batch, pages, token_ids, steps, hbm, tensor)
    if beside == "lfm2":
        out["lfm2"] = _lfm2_prefill(device, blaslt, batch, pages, token_ids, steps, hbm, tensor)
    elif beside is not None:
        out[beside.name] = _stack_prefill(device, blaslt, beside, batch, pages, token_ids, steps, hbm, tensor)
    blaslt.close()
    torch.cuda.empty_cache()
    return out


# Other sizes: for Fegidra heads of 128 with chunks shorter than the contexts, for Ribivik heads of 128 and fewer or more of
# them; one smaller and one larger width.
OTHER_SIZES = {
    "fegidra": {
        "width 1024": dict(width=1024, num_layers=8, attention_layers=(2, 5), heads=8, kv_heads=2, dim=128, delta_heads=16,
                           ff=6144, vocab=32768, chunk=512),
        "width 4096": dict(width=4096, num_layers=8, attention_layers=(2, 5), heads=32, kv_heads=8, dim=128, delta_heads=32,
                           delta_dim=128, ff=24576, vocab=65536, chunk=1024)},
    "ribivik": {
        "width 1024": dict(width=1024, num_layers=8, attention_layers=(2, 5), heads=16, dim=64, rot_dim=32, vdim=64,
                           q_rank=384, kv_rank=256, ssm_heads=32, state=64, groups=1, ff=6144, vocab=32768),
        "width 2048, heads of 128": dict(num_layers=8, attention_layers=(2, 5), heads=16, dim=128, vdim=128),
        "width 4096": dict(width=4096, num_layers=8, attention_layers=(2, 5), heads=64, dim=128, vdim=128, q_rank=1536,
                           ssm_heads=128, ff=24576)},
}
DESIGNS = {"fegidra": (fegidra_design, lambda: "lfm2"), "ribivik": (ribivik_design, fegidra_design)}


def run(device, steps: int, hbm: float, tensor: float, design_name: str = "fegidra") -> dict:
    make, beside_of = DESIGNS[design_name]
    design, beside = make(), beside_of()
    few = max(steps // 8, 4)
    with torch.cuda.stream(torch.cuda.Stream(device=device)):
        decode = [decode_case(device, sequences, contexts, steps, design, beside, hbm, tensor)
                  for sequences, contexts in ((1, (1024, 1024)), (32, (128, 4096)), (128, (128, 4096)))]
        prefill = [prefill_case(device, [0] * 8, 512, few, design, beside, hbm, tensor),
                   prefill_case(device, [0], 4096, few, design, beside, hbm, tensor),
                   prefill_case(device, [1024] * 8, 512, few, design, beside, hbm, tensor)]
        others = {}
        for name, sizes in OTHER_SIZES[design_name].items():
            other = make(**sizes)
            others[name] = {"decode": decode_case(device, 64, (128, 4096), steps, other, None, hbm, tensor),
                            "prefill": prefill_case(device, [0] * 8, 512, few, other, None, hbm, tensor)}
    return {"decode": decode, "prefill": prefill, "other_sizes": others}

"""Throughput of a layer-stack model beside the LFM2 model at equal size: decode steps and mixed prefill steps with
random weights, and the device time of every kernel of a step against its roofline.

The stack is a Fegidra of LFM2.5-1.2B's shape: width 2048, 16 layers of which the same six are attention (32 query and
8 key/value heads of 64), delta-rule layers of 32 heads of 64 in place of the gated convolutions, feed-forwards of
12288 (two matrices with as many weights as SwiGLU's three at 8192), vocabulary 65536.  Both run in BF16.
"""
from __future__ import annotations

import re

import numpy as np
import torch

from . import fegidra, ops, stack, workloads
from . import model as lfm_model

RANK = 64
TAPS = 4


def config(width=2048, num_layers=16, attention_layers=lfm_model.ATTENTION_LAYERS, heads=32, kv_heads=8, dim=64,
           delta_heads=32, delta_dim=64, ff=12288, vocab=lfm_model.VOCAB, chunk=8192) -> dict:
    attention = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk},
                 "rot": {"base": 10000.0, "dims": dim}, "scale": dim ** -0.5}
    delta = {"heads": delta_heads, "dim": delta_dim}
    return {"vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "canon": {"taps": TAPS},
            "layers": [{"type": "attention" if index in attention_layers else "general_delta",
                        "mixer": attention if index in attention_layers else delta,
                        "mlp": {"kind": "dense", "ff": ff}} for index in range(num_layers)]}


def random_model(node: dict, seed: int, device, num_pages: int, slots: int, rank: int = RANK,
                 dtype: str = "bfloat16") -> stack.StackModel:
    generator = torch.Generator(device=device).manual_seed(seed)

    def source(name, shape):
        values = torch.randn(shape, generator=generator, device=device)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            values = 1.0 + 0.1 * values
        elif name.endswith(".act"):
            values = torch.tensor([0.5, 0.3, 0.2, 0.0], device=device)
        elif len(shape) == 2:
            values = values * shape[1] ** -0.5
        else:
            values = values * 0.1
        return values.to(torch.bfloat16)

    return fegidra.build(fegidra.FegidraConfig.from_json(node), source, lambda name: (rank,), device, num_pages, slots,
                         dtype)


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


def _bytes_and_flops(node: dict, tokens: int, keys: float, segments: int) -> dict:
    """Algorithmic bytes (activations, caches and state once) and flops per launch of the stack's own kernels.  `keys`:
    visible keys summed over the tokens; cache rows are counted once per token for decode and once per segment else."""
    width, layers = node["width"], node["layers"]
    attention = next(layer["mixer"] for layer in layers if layer["type"] == "attention")
    delta = next(layer["mixer"] for layer in layers if layer["type"] == "general_delta")
    ff = layers[0]["mlp"]["ff"]
    heads, groups, dim, vdim = attention["heads"], attention["kv_heads"], attention["dim"], attention["vdim"]
    projected = heads * dim + groups * (dim + vdim)
    inner = delta["heads"] * delta["dim"]
    state = delta["heads"] * delta["dim"] ** 2 * 4
    return {
        "residual_norm_conv_kernel": (tokens * width * (4 + 2 + 4 + 2 + 2) + segments * width * (TAPS - 1) * 4, 0.0),
        "poly_norm_kernel": (tokens * ff * 4, 0.0),
        "projection_norm_rope_kernel": (tokens * projected * 4, 0.0),
        "attention": (keys * groups * (dim + vdim) * 2 if segments == tokens else 0.0,
                      2.0 * keys * heads * (dim + vdim)),
        "delta": (tokens * (6 * inner + RANK) * 2 + segments * state * 2,
                              tokens * delta["heads"] * delta["dim"] ** 2 * 10.0),
    }


def rooflines(node, times, tokens, keys, segments, hbm_gbs, tensor_tflops, fp32_tflops=75.0) -> dict:
    """Per kernel: achieved over the roofline that bounds it (delta rule: f32 multiply-adds outside the tensor cores,
    at the nominal rate)."""
    out = {}
    for kernel, (launches, micros) in times.items():
        key = next((word for word in ("attention", "delta") if word in kernel), kernel)
        work = _bytes_and_flops(node, tokens, keys, segments).get(key)
        if work is None:
            continue
        peak = fp32_tflops if key == "delta" else tensor_tflops
        ideal = max(work[0] / (hbm_gbs * 1e9), work[1] / (peak * 1e12)) * 1e6
        out[kernel] = {"us": round(micros, 2), "roofline_us": round(ideal, 2), "frac": round(ideal / micros, 3)}
    return out


def decode_case(device, sequences: int, contexts, steps: int, node: dict, hbm: float, tensor: float,
                beside_lfm2: bool = True) -> dict:
    """Decode steps replayed from their graphs, of the stack and, on the same batch, of the LFM2 model."""
    batch = workloads.ragged_decode_batch(1, sequences, contexts[0], contexts[1],
                                          sequences * (contexts[1] // 16 + 8) + 64, 64)
    token_ids = np.random.default_rng(3).integers(0, node["vocab"], size=sequences).astype(np.uint32)
    context = int(batch.contexts.max()) + 64
    out = {"sequences": sequences, "contexts": list(contexts)}

    def fixed_batch():
        return lfm_model.DecodeBatch(device, batch.block_tables, batch.request_slots, batch.positions(0), token_ids,
                                     context)

    blaslt = ops.BlasLt()
    blaslt.bind_current_stream()
    model = random_model(node, 7, device, batch.num_pages, sequences)
    executor = stack.StackExecutor(blaslt, model, sequences)
    device_batch = fixed_batch()
    milliseconds = timed_ms(lambda: executor.step_graph(device_batch, advance=False), steps)
    times = kernel_times(lambda: executor.step_graph(device_batch, advance=False))
    limit = next(layer["mixer"]["mask"]["size"] for layer in node["layers"] if layer["type"] == "attention")
    keys = float((batch.positions(0).astype(np.float64) % limit + 1).sum())
    out["stack"] = {"ms_per_step": milliseconds, "tok_s": sequences / milliseconds * 1e3,
                    "kernels": {name: [count, round(micros, 2)] for name, (count, micros) in times.items()},
                    "rooflines": rooflines(node, times, sequences, keys, sequences, hbm, tensor),
                    "launches": executor.graph_kernels(), "weight_bytes": model.weight_bytes()}
    executor.close()
    del model
    if not beside_lfm2:
        blaslt.close()
        torch.cuda.empty_cache()
        return out
    reference = lfm_model.RandomModel(7, device, batch.num_pages, sequences, fp8_policy=False)
    closest = lfm_model.DecodeExecutor(blaslt, sequences)
    device_batch = fixed_batch()
    milliseconds = timed_ms(lambda: closest.step_graph(reference, device_batch, use_fp8=False, advance=False), steps)
    times = kernel_times(lambda: closest.step_graph(reference, device_batch, use_fp8=False, advance=False))
    out["lfm2"] = {"ms_per_step": milliseconds, "tok_s": sequences / milliseconds * 1e3,
                   "kernels": {name: [count, round(micros, 2)] for name, (count, micros) in times.items()},
                   "rooflines": _lfm2_rooflines(times, sequences, keys, sequences, hbm, tensor),
                   "launches": closest.graph_kernels(), "weight_bytes": reference.weight_bytes(False)}
    closest.close()
    blaslt.close()
    del reference
    torch.cuda.empty_cache()
    return out


def _lfm2_rooflines(times, tokens, keys, segments, hbm, tensor) -> dict:
    rows = {"rms_norm_kernel": (tokens * 2048 * 8, 0.0), "short_conv": (tokens * 2048 * 8 + segments * 2048 * 8, 0.0),
            "silu_mul": (tokens * 8192 * 6, 0.0), "qk_norm_rope": (tokens * 3072 * 4, 0.0),
            "attention": (keys * 8 * 256 if segments == tokens else 0.0, 4.0 * keys * 2048)}
    out = {}
    for kernel, (_, micros) in times.items():
        work = next((work for name, work in rows.items() if name in kernel), None)
        if work is not None:
            ideal = max(work[0] / (hbm * 1e9), work[1] / (tensor * 1e12)) * 1e6
            out[kernel] = {"us": round(micros, 2), "roofline_us": round(ideal, 2), "frac": round(ideal / micros, 3)}
    return out


def prefill_case(device, prefixes, chunk: int, steps: int, node: dict, hbm: float, tensor: float,
                 beside_lfm2: bool = True) -> dict:
    """Mixed steps of `chunk` new tokens behind each of `prefixes` cached ones."""
    pages = sum((prefix + chunk + 15) // 16 for prefix in prefixes)
    batch = workloads.mixed_step_batch(5, prefixes, [chunk] * len(prefixes), pages)
    token_ids = np.random.default_rng(5).integers(0, node["vocab"], size=batch.num_tokens).astype(np.uint32)
    limit = next(layer["mixer"]["mask"]["size"] for layer in node["layers"] if layer["type"] == "attention")
    positions = batch.positions.astype(np.float64)
    out = {"prefixes": list(prefixes), "chunk": chunk, "attention_chunk": limit}
    blaslt = ops.BlasLt()
    blaslt.bind_current_stream()
    model = random_model(node, 7, device, pages, batch.num_segments)
    executor = stack.StackExecutor(blaslt, model, batch.num_tokens, batch.num_segments)
    device_batch = lfm_model.RaggedBatch(device, batch, token_ids)
    milliseconds = timed_ms(lambda: executor.forward_ragged(device_batch), steps)
    times = kernel_times(lambda: executor.forward_ragged(device_batch))
    keys = float((positions % limit + 1).sum())
    out["stack"] = {"ms_per_step": milliseconds, "tok_s": batch.num_tokens / milliseconds * 1e3,
                    "kernels": {name: [count, round(micros, 2)] for name, (count, micros) in times.items()},
                    "rooflines": rooflines(node, times, batch.num_tokens, keys, batch.num_segments, hbm, tensor)}
    executor.close()
    del model
    if not beside_lfm2:
        blaslt.close()
        torch.cuda.empty_cache()
        return out
    reference = lfm_model.RandomModel(7, device, pages, batch.num_segments, fp8_policy=False)
    closest = lfm_model.DecodeExecutor(blaslt, batch.num_tokens, maximum_segments=batch.num_segments)
    device_batch = lfm_model.RaggedBatch(device, batch, token_ids)
    milliseconds = timed_ms(lambda: closest.forward_ragged(reference, device_batch, use_fp8=False), steps)
    times = kernel_times(lambda: closest.forward_ragged(reference, device_batch, use_fp8=False))
    out["lfm2"] = {"ms_per_step": milliseconds, "tok_s": batch.num_tokens / milliseconds * 1e3,
                   "kernels": {name: [count, round(micros, 2)] for name, (count, micros) in times.items()},
                   "rooflines": _lfm2_rooflines(times, batch.num_tokens, float((positions + 1).sum()),
                                                batch.num_segments, hbm, tensor)}
    closest.close()
    blaslt.close()
    del reference
    torch.cuda.empty_cache()
    return out


# Other sizes, without a counterpart: heads of 128 with chunks shorter than the contexts, one smaller and one larger width.
OTHER_SIZES = {
    "width 1024": dict(width=1024, num_layers=8, attention_layers=(2, 5), heads=8, kv_heads=2, dim=128, delta_heads=16,
                       ff=6144, vocab=32768, chunk=512),
    "width 4096": dict(width=4096, num_layers=8, attention_layers=(2, 5), heads=32, kv_heads=8, dim=128, delta_heads=32,
                       delta_dim=128, ff=24576, vocab=65536, chunk=1024),
}


def run(device, steps: int, hbm: float, tensor: float) -> dict:
    node = config()
    few = max(steps // 8, 4)
    with torch.cuda.stream(torch.cuda.Stream(device=device)):
        decode = [decode_case(device, sequences, contexts, steps, node, hbm, tensor)
                  for sequences, contexts in ((1, (1024, 1024)), (32, (128, 4096)), (128, (128, 4096)))]
        prefill = [prefill_case(device, [0] * 8, 512, few, node, hbm, tensor),
                   prefill_case(device, [0], 4096, few, node, hbm, tensor),
                   prefill_case(device, [1024] * 8, 512, few, node, hbm, tensor)]
        others = {}
        for name, sizes in OTHER_SIZES.items():
            other = config(**sizes)
            others[name] = {"decode": decode_case(device, 64, (128, 4096), steps, other, hbm, tensor, False),
                            "prefill": prefill_case(device, [0] * 8, 512, few, other, hbm, tensor, False)}
    return {"decode": decode, "prefill": prefill, "other_sizes": others}

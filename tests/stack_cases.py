"""What the tests of all layer-stack designs share: rounding, engines, steps of one layer, error measures."""
from __future__ import annotations

import contextlib

import numpy as np


def bf16_values(values: np.ndarray) -> np.ndarray:
    """Rounded to bf16, as float64."""
    import torch
    return torch.from_numpy(np.asarray(values, dtype=np.float32)).to(torch.bfloat16).to(torch.float64).numpy()


def torch_source(tensors):
    import torch

    def source(name, shape):
        assert tensors[name].shape == tuple(shape), name
        return torch.from_numpy(tensors[name]).to(torch.bfloat16)
    return source


@contextlib.contextmanager
def engine_around(make_model, device, slots, sequence_tokens=512, prefill_tokens=512, radix_pages=1, calibrate=False):
    """A serving engine on a stream of its own around the model that `make_model` builds."""
    import torch

    from lfm25_inference_b200 import serving
    with torch.cuda.stream(torch.cuda.Stream(device)):
        engine = serving.ServingEngine(make_model(), device, max_slots=slots, max_sequence_tokens=sequence_tokens,
                                       max_prefill_tokens=prefill_tokens, radix_pages=radix_pages,
                                       checkpoint_capacity=8, use_fp8=False)
        if calibrate:
            engine.calibrate()
        try:
            yield engine
        finally:
            engine.close()


def residual_in_portions(make_model, device, tokens, portions) -> np.ndarray:
    """The residual stream behind the last layer for every token of one sequence fed in `portions` through the executor.
    `make_model(num_pages, slots)`; the sequence lives in slot 1 on pages in random order."""
    import torch

    from lfm25_inference_b200 import model as lfm_model
    from lfm25_inference_b200 import ops, stack, workloads
    got, pages, at = [], (len(tokens) + 15) // 16, 0
    with torch.cuda.stream(torch.cuda.Stream(device)):
        model = make_model(pages + 3, 2)
        blaslt = ops.BlasLt()
        executor = stack.StackExecutor(blaslt, model, len(tokens))
        table = np.random.default_rng(7).permutation(pages + 3).astype(np.uint32)[:pages].reshape(1, -1)
        table = np.concatenate([np.full_like(table, 0xFFFFFFFF), table])
        for size in portions:
            batch = workloads.MixedStepBatch(pages + 3, table, np.array([at]), np.array([size]),
                                             np.array([1], np.uint32))
            executor.forward_ragged(lfm_model.RaggedBatch(device, batch, tokens[at:at + size]))
            got.append(executor.residual(size))
            at += size
        assert ops.device_status()[0] == 0
        executor.close()
        blaslt.close()
    return np.concatenate(got)


def feed(engine, vocab, request, tokens, portions):
    """Feeds `tokens` of one request in portions of the given sizes; every token's logits."""
    rows, at = [], 0
    for size in portions:
        part = tokens[at:at + size]
        rows.append(engine.forced_step([(request, part, range(len(part)))], vocab))
        at += size
    assert at == len(tokens)
    return np.concatenate(rows)


def relative_error(got, want) -> np.ndarray:
    """Per row: RMS of the difference over the RMS of the expected rows around their means."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    centred = want - want.mean(-1, keepdims=True)
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((centred ** 2).mean())


# what rounding leaves in either activation type (the bf16 figure: a few layers of bf16 activations)
LIMITS = {"float32": 3e-5, "bfloat16": 6e-2}

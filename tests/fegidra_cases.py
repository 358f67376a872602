"""Small Fegidra configurations with random weights, and the framework driven next to the plain restatement."""
from __future__ import annotations

import contextlib

import numpy as np

from oracle import fegidra as oracle_fegidra


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, chunk=24, rot_dims=8, base=1000.0, scale=None, ff=40) -> dict:
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
                      "rot": {"dims": rot_dims, "base": base}, "scale": dim ** -0.5 if scale is None else scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta_layer(heads=3, dim=16, ff=40) -> dict:
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config_of(layers, vocab=88, width=48, taps=3, eps=1e-4) -> dict:
    return {"architecture": "Fegidra", "vocab": vocab, "width": width, "canon": {"taps": taps}, "norm": {"eps": eps},
            "layers": list(layers)}


MIXED = (attention_layer(), delta_layer(), delta_layer(heads=2, dim=24, ff=0), attention_layer(heads=6, kv_heads=3, ff=64))


def bf16_values(values: np.ndarray) -> np.ndarray:
    """Rounded to bf16, as float64."""
    import torch
    return torch.from_numpy(np.asarray(values, dtype=np.float32)).to(torch.bfloat16).to(torch.float64).numpy()


def random_tensors(config: dict, seed: int, rank: int = 5) -> dict[str, np.ndarray]:
    """bf16-representable float64 arrays under the checkpoint's names.  Norm weights away from 1, decays that differ
    between channels and removal rates of every size, so that a mixed-up vector shows."""
    from lfm25_inference_b200 import fegidra
    rng = np.random.default_rng(seed)
    tensors = {}
    for name, shape in fegidra.tensor_shapes(fegidra.FegidraConfig.from_json(config), rank).items():
        values = rng.standard_normal(shape)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            values = 1.0 + 0.3 * values
        elif name.endswith(".act"):
            values = np.array([0.6, -0.4, 0.3, 0.2])
        elif name.endswith("w0"):
            values = 2.0 * values - 2.0
        elif len(shape) == 2 and not name.startswith("embed") and "canon" not in name:
            values = values * 1.5 * shape[1] ** -0.5
        elif "canon" in name:
            values = values * 0.4
        tensors[name] = bf16_values(values)
    return tensors


def torch_source(tensors):
    import torch

    def source(name, shape):
        assert tensors[name].shape == tuple(shape), name
        return torch.from_numpy(tensors[name]).to(torch.bfloat16)
    return source


def product_model(config, tensors, device, dtype, num_pages=96, slots=8):
    from lfm25_inference_b200 import fegidra
    return fegidra.build(fegidra.FegidraConfig.from_json(config), torch_source(tensors),
                         lambda name: tensors[name].shape, device, num_pages, slots, dtype)


def oracle_model(config, tensors, dtype=np.float64):
    return oracle_fegidra.Model(config, tensors, dtype)


@contextlib.contextmanager
def engine_of(config, tensors, device, dtype, num_pages=96, slots=8, sequence_tokens=512, prefill_tokens=512,
              radix_pages=1, calibrate=False):
    """A serving engine on a stream of its own around a freshly built model."""
    import torch

    from lfm25_inference_b200 import serving
    with torch.cuda.stream(torch.cuda.Stream(device)):
        model = product_model(config, tensors, device, dtype, num_pages, slots)
        engine = serving.ServingEngine(model, device, max_slots=slots, max_sequence_tokens=sequence_tokens,
                                       max_prefill_tokens=prefill_tokens, radix_pages=radix_pages,
                                       checkpoint_capacity=8, use_fp8=False)
        if calibrate:
            engine.calibrate()
        try:
            yield engine
        finally:
            engine.close()


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

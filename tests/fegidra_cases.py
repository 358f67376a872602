"""Small Fegidra configurations with random weights, and the framework driven next to the plain restatement."""
from __future__ import annotations

import numpy as np

from oracle import fegidra as oracle_fegidra
from stack_cases import LIMITS, bf16_values, engine_around, feed, relative_error, torch_source  # noqa: F401


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


def product_model(config, tensors, device, dtype, num_pages=96, slots=8):
    from lfm25_inference_b200 import fegidra
    return fegidra.build(fegidra.FegidraConfig.from_json(config), torch_source(tensors),
                         lambda name: tensors[name].shape, device, num_pages, slots, dtype)


def oracle_model(config, tensors, dtype=np.float64):
    return oracle_fegidra.Model(config, tensors, dtype)


def engine_of(config, tensors, device, dtype, num_pages=96, slots=8, **options):
    """A serving engine around a freshly built model."""
    return engine_around(lambda: product_model(config, tensors, device, dtype, num_pages, slots), device, slots, **options)

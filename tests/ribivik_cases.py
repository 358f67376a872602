"""Small Ribivik configurations with random weights, and the framework driven next to the plain restatement."""
from __future__ import annotations

import numpy as np

from oracle import ribivik as oracle_ribivik
from stack_cases import bf16_values, engine_around, feed, relative_error, torch_source  # noqa: F401


def latent_layer(heads=3, dim=24, rot_dim=8, vdim=16, q_rank=32, kv_rank=40, base=500.0, scale=None, kv_from=None,
                 ff=56) -> dict:
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mamba_layer(heads=6, vdim=8, state=16, groups=3, norm_groups=2, conv=3, ff=0) -> dict:
    return {"type": "mamba2",
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                      "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config_of(layers, vocab=88, width=48, eps=1e-4, softcap=9.0) -> dict:
    return {"architecture": "Ribivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": softcap,
            "layers": list(layers)}


# own latents, shared ones (also across a layer with latents of its own), recurrences with and without a feed-forward
MIXED = (latent_layer(), mamba_layer(ff=40), mamba_layer(heads=2, vdim=24, state=40, groups=1, norm_groups=1),
         latent_layer(heads=2, dim=16, vdim=32, q_rank=24, kv_from=0, ff=0),
         latent_layer(heads=5, dim=40, rot_dim=24, vdim=8, kv_rank=72, base=70.0, scale=0.2),
         latent_layer(heads=4, kv_from=0, scale=0.3))


def random_tensors(config: dict, seed: int) -> dict[str, np.ndarray]:
    """bf16-representable float64 arrays under the checkpoint's names: norm weights, step sizes and decay rates that differ
    from channel to channel, so that a mixed-up vector shows."""
    from lfm25_inference_b200 import ribivik
    rng = np.random.default_rng(seed)
    tensors = {}
    for name, shape in ribivik.tensor_shapes(ribivik.RibivikConfig.from_json(config)).items():
        values = rng.standard_normal(shape)
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            values = 0.3 * values
        elif leaf == "norm":
            values = 1.0 + 0.3 * values
        elif leaf == "dt_bias":
            values = values - 2.0
        elif leaf in ("A_log", "conv", "b"):
            values = 0.7 * values
        elif len(shape) == 2 and name != "embed":
            values = values * 1.5 * shape[1] ** -0.5
        tensors[name] = bf16_values(values)
    return tensors


def product_model(config, tensors, device, dtype, num_pages=96, slots=8):
    from lfm25_inference_b200 import ribivik
    return ribivik.build(ribivik.RibivikConfig.from_json(config), torch_source(tensors), device, num_pages, slots, dtype)


def oracle_model(config, tensors, dtype=np.float64):
    return oracle_ribivik.Model(config, tensors, dtype)


def engine_of(config, tensors, device, dtype, num_pages=96, slots=8, **options):
    """A serving engine around a freshly built model."""
    return engine_around(lambda: product_model(config, tensors, device, dtype, num_pages, slots), device, slots, **options)


# What rounding leaves.  In bf16 single tokens stand out: where a sublayer's output nearly cancels, the norm behind it
# amplifies what rounding left, so the bounds on most tokens are the sharp ones.
SHARP = {"float32": 1e-4, "bfloat16": 0.3}


def assert_logits(got, want, dtype):
    error = relative_error(got, want)
    assert error.max() <= SHARP[dtype], (int(error.argmax()), float(error.max()))
    if dtype == "bfloat16":
        assert np.median(error) <= 4e-2, float(np.median(error))

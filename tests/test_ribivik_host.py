"""Host side of the Ribivik family without a GPU: the plain restatement against small hand-made cases, configuration and
tensor shapes, the registry, and what the executor refuses."""
import ctypes
import json

import numpy as np
import pytest

import ribivik_cases as cases
from lfm25_inference_b200 import _abi, cli, registry, ribivik
from lfm25_inference_b200 import model as lfm_model
from lfm25_inference_b200 import workloads
from oracle import ribivik as oracle_ribivik


# ------------------------------------------------------------------------------------------------ the restatement

def test_norm_weights_are_distances_from_one():
    x = np.array([[3.0, -4.0]])
    want = x / np.sqrt(12.5 + 0.5) * np.array([1.25, 0.5])
    assert np.allclose(oracle_ribivik.shifted_norm(x, np.array([0.25, -0.5]), 0.5), want)


def test_activations_by_hand():
    assert np.allclose(oracle_ribivik.softplus(np.array([-800.0, 0.0, 800.0])), [0.0, np.log(2.0), 800.0])
    assert oracle_ribivik.squared_relu(np.array([-3.0, 0.5])).tolist() == [0.0, 0.25]
    assert np.allclose(oracle_ribivik.softcap(np.array([1e9, 0.0, -2.0]), 4.0), [4.0, 0.0, -4.0 * np.tanh(0.5)])
    assert oracle_ribivik.softcap(np.array([70.0]), None).tolist() == [70.0]


def test_latent_scores_add_both_parts():
    """One head of one unrotated and two rotated dimensions: the score is (q k + r . s) scale, the value comes from the
    latent."""
    latents, rotated_keys = np.array([[2.0], [5.0]]), np.array([[1.0, 0.0], [0.0, 3.0]])
    keys, values = oracle_ribivik.expand(latents, np.array([[0.5]]), np.array([[10.0], [-1.0]]), 1)
    assert keys[0, :, 0].tolist() == [1.0, 2.5] and values[0].tolist() == [[20.0, -2.0], [50.0, -5.0]]
    out = oracle_ribivik.softmax_over(np.array([[4.0]]), np.array([[1.0, -1.0]]), keys, values, rotated_keys, 0.25)
    scores = 0.25 * np.array([4.0 * 1.0 + 1.0, 4.0 * 2.5 - 3.0])
    weight = np.exp(scores[1]) / np.exp(scores).sum()
    assert np.allclose(out[0], (1 - weight) * values[0, 0] + weight * values[0, 1])


def test_recurrence_step_by_hand():
    state = np.array([[1.0, 2.0], [3.0, 4.0], [0.0, -1.0]])           # [N, V]
    x, b, c = np.array([10.0, 20.0]), np.array([1.0, 0.0, 2.0]), np.array([1.0, -1.0, 0.5])
    new, y = oracle_ribivik.ssd_step(state, x, b, c, 0.5, 3.0, 7.0)
    want = np.exp(-1.5) * state + 0.5 * np.array([[10.0, 20.0], [0.0, 0.0], [20.0, 40.0]])
    assert np.allclose(new, want) and np.allclose(y, want[0] - want[1] + 0.5 * want[2] + 7.0 * x)


def test_gated_output_is_normed_part_by_part():
    y, z = np.array([[1.0, 2.0, 3.0, 4.0]]), np.array([[0.5, -1.0, 2.0, 0.0]])
    gated = y * z / (1.0 + np.exp(-z))
    want = np.concatenate([part / np.sqrt((part ** 2).mean() + 0.1) for part in (gated[0, :2], gated[0, 2:])])
    weight = np.array([1.0, 2.0, 3.0, 4.0])
    assert np.allclose(oracle_ribivik.gated_group_norm(y, z, weight, 2, 0.1)[0], want * weight)


def test_shared_latents_are_read_and_not_written():
    config = cases.config_of([cases.latent_layer(ff=0), cases.latent_layer(heads=2, kv_from=0, ff=0)])
    tensors = cases.random_tensors(config, 3)
    assert not any(name.startswith("l1.mix.dkv") for name in tensors)
    model = cases.oracle_model(config, tensors)
    state = model.new_state()
    model.forward([1, 2, 3], state)
    assert state["layers"][0][0].shape == (3, 40) and state["layers"][1][0].shape == (0, 40)


def test_restatement_does_not_depend_on_portions():
    config = cases.config_of(cases.MIXED)
    tensors = cases.random_tensors(config, 5)
    model = cases.oracle_model(config, tensors)
    tokens = np.random.default_rng(1).integers(0, config["vocab"], size=60)
    whole = model.forward(tokens, model.new_state())
    state, parts = model.new_state(), []
    for begin, end in ((0, 2), (2, 3), (3, 26), (26, 58), (58, 60)):
        parts.append(model.forward(tokens[begin:end], state))
    assert np.allclose(np.concatenate(parts), whole, atol=1e-9)


# ------------------------------------------------------------------------------------------------ configuration

def test_configuration_reads_every_size():
    config = cases.config_of([cases.latent_layer(6, 10, 4, 14, 9, 11, base=9.0, scale=0.2, ff=7),
                              cases.mamba_layer(6, 5, 3, 2, 10, 4, ff=0),
                              cases.latent_layer(3, 20, 4, 6, 5, 11, base=9.0, kv_from=0, ff=0)],
                             vocab=71, width=22, eps=1e-3, softcap=12.5)
    parsed = ribivik.RibivikConfig.from_json(json.loads(json.dumps(config)))
    assert (parsed.vocab, parsed.width, parsed.norm_eps, parsed.logit_softcap) == (71, 22, 1e-3, 12.5)
    assert parsed.layers[0].mixer == ribivik.LatentAttentionConfig(6, 10, 4, 14, 9, 11, 0.2, 4, 9.0, None)
    assert parsed.layers[0].ff == 7 and parsed.layers[2].mixer.kv_from == 0
    assert parsed.layers[1].mixer == ribivik.Mamba2Config(6, 5, 3, 2, 10, 4) and parsed.layers[1].ff == 0
    shapes = ribivik.tensor_shapes(parsed)
    assert shapes["l0.mix.uq"] == (84, 9) and shapes["l0.mix.dkv"] == (15, 22) and shapes["l0.mix.g"] == (84, 22)
    assert shapes["l1.mix.in"] == (30 + 30 + 12 + 6, 22) and shapes["l1.mix.conv"] == (42, 4)
    assert "l2.mix.dkv" not in shapes and shapes["l2.mix.uk"] == (60, 11) and "l2.norm2" not in shapes
    assert shapes["l0.norm2b"] == (22,) and shapes["head"] == (71, 22)


@pytest.mark.parametrize("damage", [
    lambda c: c.pop("width"), lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mlp"].update(kind="other"), lambda c: c["layers"][0]["mixer"].pop("scale"),
    lambda c: c["layers"][1]["mixer"].update(groups=4), lambda c: c["layers"][1]["mixer"].update(norm_groups=5),
    lambda c: c["layers"][2]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_from=1),
    lambda c: c["layers"][2]["mixer"].update(kv_rank=16), lambda c: c["layers"][3]["mixer"].update(kv_from=2)])
def test_malformed_configurations_are_refused(damage):
    config = cases.config_of([cases.latent_layer(), cases.mamba_layer(), cases.latent_layer(kv_from=0),
                              cases.latent_layer()])
    ribivik.RibivikConfig.from_json(config)
    damage(config)
    with pytest.raises(ribivik.ConfigError):
        ribivik.RibivikConfig.from_json(config)


def test_registry_and_command_line(capsys, tmp_path):
    assert registry.family_of({"architecture": "Ribivik"}).dtypes == ("bfloat16", "float32")
    assert cli.main(["models"]) == 0
    assert "Ribivik\tbfloat16, float32" in capsys.readouterr().out
    (tmp_path / "config.json").write_text(json.dumps(cases.config_of([cases.mamba_layer()])))
    assert cli.main(["info", "--model", str(tmp_path)]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"] == "Ribivik"


# ------------------------------------------------------------------------------------------------ C ABI

def test_context_rows_of_a_mixed_step():
    table = np.zeros((3, 16), np.uint32)
    batch = workloads.MixedStepBatch(1, table, np.array([9, 60, 0]), np.array([1, 5, 64]), np.array([0, 1, 2], np.uint32))
    decode, context = lfm_model.leading_decode_segments(batch)
    assert (decode, context) == (1, 10)
    assert lfm_model.prompt_context_rows(batch, decode) == 128 + 64


def latent_struct(fake):
    layer = _abi.StackLayer()
    layer.mixer, layer.heads, layer.dim, layer.vdim = _abi.MIXER_LATENT_ATTENTION, 2, 8, 8
    layer.q_rank, layer.kv_rank, layer.rot_dim = 8, 16, 4
    for name in ("mixer_norm", "mixer_post_norm", "query_latent_norm", "latent_norm", "key_cache", "value_cache"):
        setattr(layer, name, fake)
    layer.projection = _abi.StackLinear(fake, 48, 64)
    layer.query_up = _abi.StackLinear(fake, 24, 8)
    layer.latent_up = _abi.StackLinear(fake, 32, 16)
    layer.output = _abi.StackLinear(fake, 64, 16)
    return layer


def state_struct(fake):
    layer = _abi.StackLayer()
    layer.mixer, layer.heads, layer.vdim = _abi.MIXER_STATE_SPACE, 2, 8
    layer.groups, layer.state_size, layer.norm_groups, layer.conv_taps = 1, 16, 2, 4
    for name in ("mixer_norm", "mixer_post_norm", "conv", "conv_bias", "step_bias", "log_rate", "skip", "head_norm"):
        setattr(layer, name, fake)
    layer.projection = _abi.StackLinear(fake, 80, 64)
    layer.output = _abi.StackLinear(fake, 64, 16)
    layer.state_offset = 512
    return layer


@pytest.mark.parametrize("make,change,message", [
    (latent_struct, dict(kv_rank=0), "latent attention sizes"),
    (latent_struct, dict(rot_dims=6), "rotary dimensions"),
    (latent_struct, dict(latent_norm=None), "latent attention tensors"),
    (latent_struct, dict(latent_up=(31, 16)), "latent attention shapes"),
    (latent_struct, dict(projection=(47, 64)), "projection shape"),
    (latent_struct, dict(mixer_post_norm=None), "missing norms"),
    (latent_struct, dict(ff=8), "missing feed-forward weights"),
    (state_struct, dict(groups=3), "state-space sizes"),
    (state_struct, dict(norm_groups=3), "state-space sizes"),
    (state_struct, dict(state_size=4096), "state-space sizes"),
    (state_struct, dict(skip=None), "state-space tensors"),
    (state_struct, dict(conv_taps=0), "missing convolution"),
    (state_struct, dict(state_offset=1 << 20), "recurrent state outside the record"),
])
def test_stack_executor_rejects_bad_layers_before_touching_the_device(make, change, message):
    library, out, fake = _abi.library(), ctypes.c_void_p(), 0x1000
    layer = make(fake)
    for name, value in change.items():
        setattr(layer, name, _abi.StackLinear(fake, *value) if isinstance(value, tuple) else value)
    layers = (_abi.StackLayer * 1)(layer)
    model = _abi.StackModel(1, layers, _abi.ACTIVATION_BF16, _abi.BLOCK_SANDWICH, 10, 64, 1e-5, 1.0, 0.0, fake, fake,
                            _abi.StackLinear(fake, 16, 64), fake, 1 << 16, 1, 1)
    code = library.lfm25_stack_executor_create(fake, ctypes.byref(model), 8, 8, ctypes.byref(out))
    assert (code, library.lfm25_last_error().decode()) == (_abi.ERR_INVALID_ARGUMENT, f"layer 0: {message}")

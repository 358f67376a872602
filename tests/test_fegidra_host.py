"""Host side of the Fegidra family without a GPU: the plain restatement against small hand-made cases, configuration and
checkpoint handling, the model registry, the trace replay's protocol and the layout of the C structs."""
import ctypes
import io
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import fegidra_cases as cases
from lfm25_inference_b200 import _abi, checkpoint, cli, fegidra, registry, trace_runner
from oracle import fegidra as oracle_fegidra

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------------------------------------ the restatement

def test_delta_step_by_hand():
    state = np.array([[1.0, 2.0], [3.0, 4.0]])                       # [key, value]
    k, v, r = np.array([3.0, 4.0]), np.array([10.0, 20.0]), np.array([1.0, -1.0])
    decay, removal = np.array([0.5, 0.25]), np.array([1.0, 0.5])
    new, out = oracle_fegidra.delta_step(state, r, k, v, decay, removal)
    unit = k / np.sqrt(25.0 + 1e-6)
    recalled = unit[0] * state[0] + unit[1] * state[1]
    want = np.stack([decay[i] * state[i] - removal[i] * unit[i] * recalled + k[i] * v for i in range(2)])
    assert np.allclose(new, want) and np.allclose(out, want[0] - want[1])


def test_decay_range():
    h = np.random.default_rng(0).standard_normal((50, 4)) * 30
    decay = oracle_fegidra.delta_decay(h, np.eye(4), np.eye(4) * 50, np.zeros(4))
    assert decay.max() <= 1.0 and decay.min() >= np.exp(-np.exp(-0.5)) - 1e-12


def test_chunks_count_from_the_start_of_the_sequence():
    assert oracle_fegidra.visible(9, 5, 5) and not oracle_fegidra.visible(9, 4, 5)
    assert not oracle_fegidra.visible(10, 9, 5) and oracle_fegidra.visible(10, 10, 5)
    assert not oracle_fegidra.visible(3, 4, 5) and oracle_fegidra.visible(1000, 0, 0)


def test_rotation_by_hand():
    x = np.arange(1.0, 7.0).reshape(1, 1, 6)
    out = oracle_fegidra.rotate_half(x, np.array([2]), 16.0, 4)[0, 0]
    for i, angle in ((0, 2.0), (1, 2.0 * 16.0 ** -0.5)):
        u, v = x[0, 0, i], x[0, 0, i + 2]
        assert np.isclose(out[i], u * np.cos(angle) - v * np.sin(angle))
        assert np.isclose(out[i + 2], v * np.cos(angle) + u * np.sin(angle))
    assert np.array_equal(out[4:], x[0, 0, 4:])


def test_convolution_by_hand():
    h = np.array([[1.0], [2.0], [3.0]])
    out, history = oracle_fegidra.causal_convolution(h, np.array([[100.0, 10.0, 1.0]]), np.array([[7.0], [8.0]]))
    assert out[:, 0].tolist() == [781.0, 812.0, 123.0] and history[:, 0].tolist() == [2.0, 3.0]


def test_poly_norm_by_hand():
    z = np.array([[1.0, -2.0, 3.0]])
    parts = [z ** n / np.sqrt(np.mean(z ** (2 * n)) + 0.1) for n in (1, 2, 3)]
    want = 2 * parts[0] - parts[1] + 0.5 * parts[2] + 0.25
    assert np.allclose(oracle_fegidra.poly_norm(z, (2.0, -1.0, 0.5, 0.25), 0.1), want)


def test_attention_groups_and_scale():
    q, k = np.zeros((1, 4, 2)), np.zeros((2, 2, 2))
    v = np.arange(8.0).reshape(2, 2, 2)
    k[0, 1] = [1.0, 0.0]
    q[0, 2] = [2.0, 0.0]                                             # query head 2 uses key head 1
    out = oracle_fegidra.softmax_attention(q, k, v, [1], 0.5, 0)
    weight = np.exp(1.0) / (np.exp(1.0) + 1.0)
    assert np.allclose(out[0, 2], weight * v[0, 1] + (1 - weight) * v[1, 1])
    assert np.allclose(out[0, 0], v[:, 0].mean(0)) and np.allclose(out[0, 3], v[:, 1].mean(0))


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
    config = cases.config_of([cases.attention_layer(6, 2, 10, 14, 33, 4, base=9.0, scale=0.2, ff=7),
                              cases.delta_layer(5, 12, ff=0)], vocab=71, width=22, taps=6, eps=1e-3)
    parsed = fegidra.FegidraConfig.from_json(json.loads(json.dumps(config)))
    assert (parsed.vocab, parsed.width, parsed.taps, parsed.norm_eps) == (71, 22, 6, 1e-3)
    assert parsed.layers[0].mixer == fegidra.AttentionConfig(6, 2, 10, 14, 0.2, 4, 9.0, 33) and parsed.layers[0].ff == 7
    assert parsed.layers[1].mixer == fegidra.GeneralDeltaConfig(5, 12) and parsed.layers[1].ff == 0
    shapes = fegidra.tensor_shapes(parsed, 3)
    assert shapes["l0.mix.q"] == (60, 22) and shapes["l0.mix.v"] == (28, 22) and shapes["l0.mix.o"] == (22, 84)
    assert shapes["l1.mix.w2"] == (60, 3) and shapes["l1.canon1"] == (22, 6) and "l1.norm2" not in shapes


@pytest.mark.parametrize("damage", [lambda c: c.pop("width"), lambda c: c["layers"][0].update(type="other"),
                                    lambda c: c["layers"][0]["mlp"].update(kind="other"),
                                    lambda c: c["layers"][0]["mixer"].pop("scale")])
def test_malformed_configurations_are_refused(damage):
    config = cases.config_of([cases.attention_layer()])
    damage(config)
    with pytest.raises(fegidra.ConfigError):
        fegidra.FegidraConfig.from_json(config)


def test_registry_chooses_by_architecture(tmp_path):
    assert registry.family_of({"architecture": "Fegidra"}).dtypes == ("bfloat16", "float32")
    with pytest.raises(registry.UnknownModel):
        registry.family_of({"architecture": "unheard of"})
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Lfm2Random"}))
    with pytest.raises(registry.UnsupportedType):
        registry.load_model(str(tmp_path), None, 1, 1, "float32")


# ------------------------------------------------------------------------------------------------ checkpoints

def test_checkpoint_round_trip(tmp_path):
    path = str(tmp_path / "model.safetensors")
    tensors = {"a": torch.randn(3, 5).to(torch.bfloat16), "b.c": torch.arange(4, dtype=torch.int32),
               "d": torch.randn(2, 2, 2)}
    checkpoint.write(path, tensors)
    read = checkpoint.Checkpoint(path)
    assert read.names() == set(tensors) and read.shape("a") == (3, 5)
    for name, tensor in tensors.items():
        assert torch.equal(read.tensor(name), tensor) and read.tensor(name).dtype == tensor.dtype
    with pytest.raises(checkpoint.CheckpointError):
        read.tensor("missing")
    with pytest.raises(checkpoint.CheckpointError):
        read.tensor("a", (5, 3))
    (tmp_path / "broken").write_bytes(b"\x05\x00")
    with pytest.raises(checkpoint.CheckpointError):
        checkpoint.Checkpoint(str(tmp_path / "broken"))


# ------------------------------------------------------------------------------------------------ trace replay

class FakeEngine:
    """Answers every wanted place with (request number, tokens seen so far, token)."""

    def __init__(self):
        self.seen, self.ended = {}, []

    def forced_step(self, entries, vocab):
        rows = []
        for number, tokens, wanted in entries:
            base = self.seen.get(number, 0)
            rows += [[number, base + place, tokens[place]] for place in wanted]
            self.seen[number] = base + len(tokens)
        return np.asarray(rows, dtype=np.float32).reshape(-1, vocab)

    def end_forced(self, number):
        self.ended.append(number)
        del self.seen[number]


def test_replay_protocol(tmp_path):
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": [9], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": [4, 3], "want": [1, 0]},
                                     {"id": "x", "tokens": [8], "want": [0]}], "end": ["x"]},
             {"step": 5, "entries": [{"id": "x", "tokens": [1, 2], "want": [1]}], "end": ["x", "y"]}]
    answer, engine = io.StringIO(), FakeEngine()
    trace_runner.replay(engine, 3, [json.dumps(step) + "\n" for step in steps], str(tmp_path), answer)
    assert answer.getvalue().splitlines() == ["done 0", "done 1", "done 2", "done 5"]

    def rows(step):
        return np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(-1, 3).tolist()

    assert rows(0) == [[0, 0, 5], [0, 2, 7]] and not (tmp_path / "1.f32").exists()
    assert rows(2) == [[1, 2, 3], [1, 1, 4], [0, 3, 8]]              # in the order of the entries and of `want`
    assert rows(5) == [[2, 1, 2]]                                    # a new request under an old name starts over
    assert len(engine.ended) == 3 and not engine.seen


def test_command_line(capsys, tmp_path):
    assert cli.main(["models"]) == 0
    assert "Fegidra\tbfloat16, float32" in capsys.readouterr().out
    (tmp_path / "config.json").write_text(json.dumps(cases.config_of([cases.delta_layer()])))
    assert cli.main(["info", "--model", str(tmp_path)]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"] == "Fegidra"
    for name in ("trace_run", "lfm25"):
        assert os.access(os.path.join(ROOT, "bin", name), os.X_OK)


# ------------------------------------------------------------------------------------------------ C ABI

def test_struct_layouts_match_the_header(tmp_path):
    pairs = {"lfm25_stack_linear": _abi.StackLinear, "lfm25_stack_layer": _abi.StackLayer,
             "lfm25_stack_model": _abi.StackModel, "lfm25_forced_entry": _abi.ForcedEntry}
    lines = ["#include <stddef.h>", "#include <stdio.h>", '#include "lfm25_b200.h"', "int main(void) {"]
    for name, struct in pairs.items():
        lines.append(f'printf("{name} %zu\\n", sizeof({name}));')
        lines += [f'printf("{name}.{field[0]} %zu\\n", offsetof({name}, {field[0]}));' for field in struct._fields_]
    source = tmp_path / "layout.c"
    source.write_text("\n".join(lines + ["return 0; }"]))
    binary = str(tmp_path / "layout")
    subprocess.run(["gcc", "-std=c11", "-I", os.path.join(ROOT, "include"), str(source), "-o", binary], check=True)
    reported = dict(line.split() for line in subprocess.run([binary], capture_output=True, text=True,
                                                            check=True).stdout.splitlines())
    for name, struct in pairs.items():
        assert int(reported[name]) == ctypes.sizeof(struct)
        for field in struct._fields_:
            assert int(reported[f"{name}.{field[0]}"]) == getattr(struct, field[0]).offset, (name, field[0])


def test_stack_executor_rejects_bad_models_before_touching_the_device():
    library = _abi.library()
    out, fake = ctypes.c_void_p(), 0x1000
    layer = _abi.StackLayer()
    layer.mixer, layer.mixer_norm, layer.conv, layer.heads, layer.dim = _abi.MIXER_GENERAL_DELTA, fake, fake, 2, 300
    layer.projection = _abi.StackLinear(fake, 3200, 64)
    layer.output = _abi.StackLinear(fake, 64, 600)
    layer.conv_taps = 2
    layers = (_abi.StackLayer * 1)(layer)
    model = _abi.StackModel(1, layers, _abi.ACTIVATION_BF16, _abi.BLOCK_PARALLEL, 10, 64, 1e-5, 0.0, 0.0, fake, fake,
                            _abi.StackLinear(fake, 16, 64), fake, 1 << 20, 1, 1)

    def create(tokens=8, rows=8):
        code = library.lfm25_stack_executor_create(fake, ctypes.byref(model), tokens, rows, ctypes.byref(out))
        return code, library.lfm25_last_error().decode()

    assert create() == (_abi.ERR_INVALID_ARGUMENT, "layer 0: delta-rule head size beyond 256")
    layers[0].dim = 0
    assert create() == (_abi.ERR_INVALID_ARGUMENT, "layer 0: mixer without heads")
    layers[0].dim, layers[0].mixer = 300, 7
    assert create() == (_abi.ERR_INVALID_ARGUMENT, "layer 0: unknown mixer")
    assert create(tokens=4, rows=8)[0] == _abi.ERR_INVALID_ARGUMENT
    model.head = _abi.StackLinear(fake, 8, 64)
    assert create() == (_abi.ERR_INVALID_ARGUMENT, "stack model sizes are inconsistent")

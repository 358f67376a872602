"""Fegidra in the framework against the plain restatement in float64: each mechanism alone in one-layer models, whole
models in portions of every kind, mixed batches, reused pages and slots, chunk edges and far keys, and generation
through the serving engine."""
import numpy as np
import pytest

import fegidra_cases as cases
import stack_cases
from oracle import fegidra as oracle_fegidra

pytestmark = pytest.mark.gpu

TYPES = ("float32", "bfloat16")


def run_layer(config, tensors, device, dtype, portions, seed=3):
    """Residual stream behind a one-layer model's layer, framework and restatement."""
    tokens = np.random.default_rng(seed).integers(0, config["vocab"], size=sum(portions)).astype(np.uint32)
    want = []
    cases.oracle_model(config, tensors).forward(tokens, cases.oracle_model(config, tensors).new_state(), want)
    got = stack_cases.residual_in_portions(
        lambda pages, slots: cases.product_model(config, tensors, device, dtype, pages, slots), device, tokens, portions)
    return got, want[-1]


def check_layer(config, seed, device, dtype, portions, rank=5, change=None):
    tensors = cases.random_tensors(config, seed, rank)
    if change is not None:
        change(tensors)
    got, want = run_layer(config, tensors, device, dtype, portions)
    error = cases.relative_error(got, want)
    assert error.max() <= {"float32": 5e-6, "bfloat16": 2e-2}[dtype], (int(error.argmax()), float(error.max()))


# ------------------------------------------------------------------------------------------------ mechanisms alone

ATTENTION_SHAPES = [   # heads, kv_heads, dim, vdim, rot_dims, chunk
    (4, 2, 16, 24, 8, 24),          # sizes below one tensor-core chunk
    (8, 2, 64, 64, 64, 48),
    (6, 3, 96, 80, 32, 40),         # sizes that are no multiple of 64
    (5, 1, 128, 128, 16, 33),
    (3, 3, 256, 8, 128, 100),
    (2, 1, 200, 104, 2, 7),         # chunks shorter than a page
    (40, 2, 32, 16, 32, 64),        # a group beyond the decode kernel's rows
    (2, 2, 20, 12, 6, 30),          # rows without 16-byte alignment: the scalar kernel
    (1, 1, 320, 160, 64, 50),       # sizes beyond the tensor-core kernels
    (2, 1, 64, 32, 64, 1),          # every token alone
]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", ATTENTION_SHAPES, ids=lambda shape: "x".join(map(str, shape)))
def test_attention_layer(device, dtype, shape):
    heads, kv_heads, dim, vdim, rot_dims, chunk = shape
    config = cases.config_of([cases.attention_layer(heads, kv_heads, dim, vdim, chunk, rot_dims, ff=0)])
    check_layer(config, 11, device, dtype, [75, 2, 1, 50, 1, 1])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads,dim,rank", [(3, 16, 5), (2, 64, 16), (1, 24, 1), (2, 128, 33), (1, 80, 3), (2, 160, 8),
                                            (1, 256, 64), (1, 10, 7), (2, 128, 700)])
def test_delta_rule_layer(device, dtype, heads, dim, rank):
    config = cases.config_of([cases.delta_layer(heads, dim, ff=0)])
    check_layer(config, 13, device, dtype, [37, 2, 1, 16, 1, 5], rank)


@pytest.mark.parametrize("heads,dim,rank", [(3, 16, 5), (2, 64, 16), (1, 24, 1), (2, 48, 70), (1, 128, 40), (2, 64, 250)])
def test_delta_rule_prompt_kernels_agree(device, library_option, heads, dim, rank):
    """The tensor-core chunks, the token-by-token prompt kernel and the general kernel on the same bf16 inputs: all keep
    32-bit accuracy in the recurrence, so they differ by rounding of the bf16 output only.  Strong decays (the chunks
    divide by their product) and weak ones side by side, portions that end inside a tile."""
    config = cases.config_of([cases.delta_layer(heads, dim, ff=0)])
    tensors = cases.random_tensors(config, 83, rank)
    tensors["l0.mix.w0"][::2] = 9.0                # decay exp(-exp(-1/2)) throughout
    results = []
    for forced in (0, 1, 2):
        library_option("delta_prompt", forced)
        results.append(run_layer(config, tensors, device, "bfloat16", [200, 33, 2, 16, 3])[0])
    for other in results[1:]:
        assert cases.relative_error(other, results[0]).max() < 4e-3


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("width,ff", [(48, 40), (256, 72), (64, 1000), (50, 30), (96, 9)])
def test_feed_forward(device, dtype, width, ff):
    """The mixer's output projection is zero: only PolyNorm is left."""
    config = cases.config_of([cases.delta_layer(1, 16, ff=ff)], width=width)

    def only_feed_forward(tensors):
        tensors["l0.mix.o"][:] = 0.0
    check_layer(config, 17, device, dtype, [9, 2, 1], change=only_feed_forward)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 7, 13])
def test_input_convolution(device, dtype, taps):
    """Portions shorter than the history, so that old inputs move through the record."""
    config = cases.config_of([cases.delta_layer(2, 16, ff=0)], taps=taps)
    check_layer(config, 19, device, dtype, [1, 2, 1, 3, 20, 2, 1, 1])


def test_stored_activation_types_agree_on_rounding(device, library_option):
    """bf16 attention on the tensor cores against the scalar kernel on the same inputs: both keep scores and weights in
    f32, so they differ by rounding of the bf16 output only."""
    results = []
    for forced in (0, 1):
        library_option("stack_attention", forced)
        config = cases.config_of([cases.attention_layer(8, 2, 64, 64, 96, 32, scale=0.4, ff=0)])
        tensors = cases.random_tensors(config, 23)
        results.append(run_layer(config, tensors, device, "bfloat16", [130, 1, 70, 1, 1])[0])
    assert cases.relative_error(results[0], results[1]).max() < 4e-3


# ------------------------------------------------------------------------------------------------ whole models

def expected_logits(config, tensors, tokens):
    model = cases.oracle_model(config, tensors)
    return model.forward(tokens, model.new_state())


@pytest.fixture(scope="module")
def mixed_case():
    config = cases.config_of(cases.MIXED)
    tensors = cases.random_tensors(config, 29)
    tokens = np.random.default_rng(31).integers(0, config["vocab"], size=150)
    return config, tensors, tokens, expected_logits(config, tensors, tokens)


PORTIONS = {"whole": [150], "tokens": [1] * 150, "pairs": [2] * 75, "threes": [3] * 50,
            "page": [16] * 9 + [6], "edges": [15, 1, 2, 6, 23, 1, 2, 22, 25, 3, 50], "tail": [118] + [1] * 32}


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("portions", PORTIONS.values(), ids=PORTIONS.keys())
def test_portions(device, dtype, portions, mixed_case):
    config, tensors, tokens, want = mixed_case
    with cases.engine_of(config, tensors, device, dtype) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, portions)
    assert cases.relative_error(got, want).max() <= cases.LIMITS[dtype]


@pytest.mark.parametrize("dtype", TYPES)
def test_unequal_requests_in_one_step_and_reused_slots(device, dtype, mixed_case):
    """Requests of different lengths advance together, end at different times and leave their pages and slots to later
    ones; every request gives the logits it gives alone."""
    config, tensors, _, _ = mixed_case
    rng = np.random.default_rng(37)
    lengths = [70, 1, 33, 16, 97, 2, 50, 49, 17, 64]
    prompts = [rng.integers(0, config["vocab"], size=length) for length in lengths]
    want = [expected_logits(config, tensors, prompt) for prompt in prompts]
    at, waiting, live, got = [0] * len(prompts), list(range(len(prompts))), [], [[] for _ in prompts]
    # four slots and barely enough pages: both are used again
    with cases.engine_of(config, tensors, device, dtype, num_pages=20, slots=4, sequence_tokens=128) as engine:
        while waiting or live:
            while waiting and len(live) < 4:
                live.append(waiting.pop(0))
            entries, pages = [], 20 - sum((at[i] + 15) // 16 for i in live)
            for index in live:
                size = min(int(rng.choice([1, 1, 2, 5, 31])), lengths[index] - at[index])
                need = (at[index] + size + 15) // 16 - (at[index] + 15) // 16
                if need > pages:
                    continue
                pages -= need
                entries.append((index, prompts[index][at[index]:at[index] + size], range(size)))
            logits, row = engine.forced_step(entries, config["vocab"]), 0
            for index, part, _ in entries:
                got[index].append(logits[row:row + len(part)])
                row += len(part)
                at[index] += len(part)
                if at[index] == lengths[index]:
                    engine.end_forced(index)
                    live.remove(index)
        pool = engine.snapshot()["pool"]
        assert pool["free_pages"] == pool["total_pages"] and engine.active() == 0
    for index in range(len(prompts)):
        error = cases.relative_error(np.concatenate(got[index]), want[index])
        assert error.max() <= cases.LIMITS[dtype], (index, int(error.argmax()), float(error.max()))


@pytest.mark.parametrize("dtype", TYPES)
def test_selected_places_only(device, dtype, mixed_case):
    config, tensors, tokens, want = mixed_case
    with cases.engine_of(config, tensors, device, dtype) as engine:
        assert engine.forced_step([(1, tokens[:40], [])], config["vocab"]).shape == (0, config["vocab"])
        places = [0, 1, 7, 8, 90, 109]
        got = engine.forced_step([(1, tokens[40:], places)], config["vocab"])
    assert cases.relative_error(got, want[[40 + place for place in places]]).max() <= cases.LIMITS[dtype]


def test_steps_larger_than_the_engine_are_cut(device, mixed_case):
    config, tensors, tokens, want = mixed_case
    with cases.engine_of(config, tensors, device, "float32", slots=2, prefill_tokens=30) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, [150])
    assert cases.relative_error(got, want).max() <= cases.LIMITS["float32"]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("sizes", [
    dict(vocab=101, width=40, taps=1, eps=1e-6),
    dict(vocab=640 + 8, width=72, taps=5, eps=1e-3),
    dict(vocab=33, width=30, taps=2, eps=1e-5),        # width without 16-byte rows
    dict(vocab=256, width=128, taps=4, eps=1e-5),      # shapes the tensor-core GEMMs take
], ids=lambda sizes: f"{sizes['vocab']}-{sizes['width']}-{sizes['taps']}")
def test_other_sizes(device, dtype, sizes):
    layers = [cases.delta_layer(5, 8, ff=24), cases.attention_layer(9, 3, 24, 40, 11, 4, base=77.0, scale=0.3, ff=0),
              cases.delta_layer(1, 128, ff=136), cases.attention_layer(2, 1, 8, 8, 1000, 8, ff=8)]
    config = cases.config_of(layers, **sizes)
    tensors = cases.random_tensors(config, 41, rank=9)
    tokens = np.random.default_rng(43).integers(0, config["vocab"], size=60)
    with cases.engine_of(config, tensors, device, dtype) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, [29, 2, 1, 12, 1, 15])
    assert cases.relative_error(got, expected_logits(config, tensors, tokens)).max() <= cases.LIMITS[dtype]


@pytest.mark.parametrize("dtype", TYPES)
def test_long_decoding_across_chunks(device, dtype, mixed_case):
    config, tensors, _, _ = mixed_case
    tokens = np.random.default_rng(47).integers(0, config["vocab"], size=420)
    want = expected_logits(config, tensors, tokens)
    with cases.engine_of(config, tensors, device, dtype) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, [20] + [1] * 400)
    assert cases.relative_error(got, want).max() <= cases.LIMITS[dtype]


# ------------------------------------------------------------------------------------------------ keys that stand out

def standout_model(chunk, kv_heads=2):
    """One attention layer in which the query of token 0 is the key of token 1 in every head, with a scale that lets a
    visible token 1 outweigh everything else token 0 sees."""
    config = cases.config_of([cases.attention_layer(4, kv_heads, 64, 32, chunk, 4, base=1e6, scale=0.3, ff=0)], vocab=120,
                             width=128, taps=2)
    tensors = cases.random_tensors(config, 53)
    for name in ("q", "k"):
        tensors[f"l0.mix.{name}.norm"][:] = 1.0
        tensors[f"l0.mix.{name}.b"][:] = 0.0
    tensors["l0.canon1"][:] = 0.0
    query, key = (oracle_fegidra.rms_norm(tensors["embed"][token], tensors["l0.norm1"], config["norm"]["eps"])
                  for token in (0, 1))
    keys = (tensors["l0.mix.k"] @ key).reshape(kv_heads, 64)
    wanted = np.repeat(keys, 4 // kv_heads, axis=0).reshape(-1)        # query head h reads key head h / group
    weight = tensors["l0.mix.q"]
    tensors["l0.mix.q"] = cases.bf16_values(weight + np.outer(wanted - weight @ query, query) / (query @ query))
    return config, tensors


CHUNK = 48


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("decoded", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("key,query", [
    (0, CHUNK - 1), (0, CHUNK), (CHUNK - 1, CHUNK), (CHUNK, 2 * CHUNK - 1), (CHUNK, 2 * CHUNK), (CHUNK - 1, 2 * CHUNK - 1),
    (2 * CHUNK, 2 * CHUNK + 1), (15, 16), (16, 47), (31, 32), (63, 64), (1, 40), (95, 95 + 1), (96, 143), (97, 130)])
def test_far_keys_and_chunk_edges(device, dtype, decoded, key, query):
    """Token 1 stands at `key` only, token 0 asks at the end.  The restatement itself proves that the case is sharp: hiding or
    showing that key moves the answer far beyond the limit."""
    config, tensors = standout_model(CHUNK)
    rng = np.random.default_rng(59)
    tokens = rng.integers(2, config["vocab"], size=query + 1)
    tokens[query] = 0
    other = tokens.copy()                         # the same with an ordinary token at `key`
    tokens[key] = 1
    want = expected_logits(config, tensors, tokens)[-1:]
    moved = cases.relative_error(expected_logits(config, tensors, other)[-1:], want).max()
    if key // CHUNK == query // CHUNK:
        assert moved > 3 * cases.LIMITS[dtype]
    else:
        assert moved == 0.0
    with cases.engine_of(config, tensors, device, dtype) as engine:
        portions = [query, 1] if decoded else [key + 1, query - key] if query - key > 1 else [query + 1]
        got = cases.feed(engine, config["vocab"], 1, tokens, portions)[-1:]
    assert cases.relative_error(got, want).max() <= cases.LIMITS[dtype]


@pytest.mark.parametrize("dtype", TYPES)
def test_state_reaches_far_back(device, dtype):
    """Decays close to one and one key that outweighs the rest: what the first token wrote is still read 200 tokens on,
    across portions and decoding."""
    config = cases.config_of([cases.delta_layer(2, 32, ff=0)], vocab=60, width=64, taps=2)
    tensors = cases.random_tensors(config, 61)
    tensors["l0.mix.w0"][:] = -12.0               # decay exp(-0.6 sigmoid(-12 + ...)): next to nothing is lost
    tensors["l0.mix.w2"][:] *= 0.1
    tensors["l0.mix.a.b"][:] = -12.0
    tensors["l0.mix.a"][:] *= 0.1
    tokens = np.random.default_rng(67).integers(1, config["vocab"], size=200)
    tokens[0] = 0
    other = tokens.copy()
    other[0] = 1
    want = expected_logits(config, tensors, tokens)
    moved = cases.relative_error(expected_logits(config, tensors, other)[-1:], want[-1:]).max()
    assert moved > 20 * cases.LIMITS["float32"]
    with cases.engine_of(config, tensors, device, dtype) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, [3, 64, 1, 1, 100, 1, 30])
    assert cases.relative_error(got, want).max() <= cases.LIMITS[dtype]


# ------------------------------------------------------------------------------------------------ serving

def greedy_with_margin(config, tensors, prompt, count):
    """The restatement's greedy tokens, and how far each was ahead of the runner-up."""
    model = cases.oracle_model(config, tensors)
    state = model.new_state()
    logits, out, margins = model.forward(prompt, state)[-1], [], []
    for _ in range(count):
        order = np.argsort(logits)
        out.append(int(order[-1]))
        margins.append(logits[order[-1]] - logits[order[-2]])
        logits = model.forward([out[-1]], state)[-1]
    return out, margins


def test_greedy_generation_through_the_engine(device, mixed_case):
    """The engine's own scheduler, admission, mixed steps, captured decode steps and sampling."""
    from lfm25_inference_b200 import serving
    config, tensors, _, _ = mixed_case
    rng = np.random.default_rng(71)
    prompts = [rng.integers(0, config["vocab"], size=length) for length in (5, 40, 17, 90, 1, 33, 64)]
    with cases.engine_of(config, tensors, device, "float32", slots=3, sequence_tokens=160, prefill_tokens=64,
                         calibrate=True) as engine:
        got = serving.generate(engine, prompts, 24)
        stats = engine.snapshot()["stats"]
    assert stats["mixed_steps"] > 0 and stats["decode_steps"] > 0
    for prompt, tokens in zip(prompts, got):
        want, margins = greedy_with_margin(config, tensors, prompt, 24)
        sure = next((i for i, margin in enumerate(margins) if margin < 1e-3), len(want))
        assert tokens[:sure] == want[:sure] and sure > 4


def test_shared_prefixes_restore_state_and_pages(device, mixed_case):
    """A prompt whose beginning was served before takes its pages from the index and its convolution histories and
    recurrent states from the checkpoint."""
    from lfm25_inference_b200 import serving
    config, tensors, _, _ = mixed_case
    rng = np.random.default_rng(73)
    shared = rng.integers(0, config["vocab"], size=48)
    prompts = [np.concatenate([shared, rng.integers(0, config["vocab"], size=length)]) for length in (1, 9, 21)]
    with cases.engine_of(config, tensors, device, "float32", radix_pages=32, prefill_tokens=64,
                         calibrate=True) as engine:
        tokens, reused = [], []
        for index, prompt in enumerate(prompts):
            record = serving.run_trace(engine, [serving.Request(index, prompt.astype(np.uint32), 12, 0)])["requests"][0]
            tokens.append(record["tokens"])
            reused.append(record["reused_tokens"])
    assert reused[0] == 0 and reused[1] >= 48 and reused[2] >= 48
    for prompt, produced in zip(prompts, tokens):
        want, margins = greedy_with_margin(config, tensors, prompt, 12)
        sure = next((i for i, margin in enumerate(margins) if margin < 1e-3), len(want))
        assert produced[:sure] == want[:sure] and sure > 2


def test_captured_steps_match_eager_ones(device, mixed_case):
    import torch

    from lfm25_inference_b200 import model as lfm_model
    from lfm25_inference_b200 import ops, stack, workloads
    config, tensors, _, _ = mixed_case
    batch = workloads.ragged_decode_batch(3, 5, 3, 90, 64, 8)
    token_ids = np.random.default_rng(5).integers(0, config["vocab"], size=5).astype(np.uint32)
    produced = []
    with torch.cuda.stream(torch.cuda.Stream(device)):
        for graph in (False, True):
            model = cases.product_model(config, tensors, device, "bfloat16", num_pages=64, slots=5)
            for key, value in model.caches:
                generator = torch.Generator(device=device).manual_seed(9)
                key.copy_(torch.randn(key.shape, generator=generator, device=device))
                value.copy_(torch.randn(value.shape, generator=generator, device=device))
            blaslt = ops.BlasLt()
            executor = stack.StackExecutor(blaslt, model, 8)
            device_batch = lfm_model.DecodeBatch(device, batch.block_tables, batch.request_slots, batch.positions(0),
                                                 token_ids, int(batch.contexts.max()) + 8)
            rows = []
            for step in range(6):
                if graph:
                    executor.step_graph(device_batch, advance=step > 0)
                else:
                    executor.forward(device_batch, advance=step > 0)
                rows.append(executor.logits(5))
            produced.append(np.stack(rows))
            if graph:
                assert executor.graph_captures() == 1 and executor.graph_kernels() > 0
            executor.close()
            blaslt.close()
    assert np.array_equal(produced[0], produced[1])


def test_command_line_and_trace_replay(device, mixed_case, tmp_path):
    """A model folder through the two programs, each in a process of its own."""
    import json
    import os
    import subprocess
    import sys

    import torch

    from lfm25_inference_b200 import checkpoint
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    config, tensors, tokens, want = mixed_case
    (tmp_path / "config.json").write_text(json.dumps(config))
    checkpoint.write(str(tmp_path / "model.safetensors"),
                     {name: torch.from_numpy(values).to(torch.bfloat16) for name, values in tensors.items()})

    def run(program, *arguments, **options):
        done = subprocess.run([sys.executable, os.path.join(root, "bin", program), *arguments], capture_output=True,
                              text=True, timeout=300, **options)
        assert done.returncode == 0, done.stderr[-2000:]
        return done.stdout

    prompts = [tokens[:9], tokens[20:61]]
    produced = run("lfm25", "generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "8",
                   *[word for prompt in prompts for word in ("--tokens", ",".join(map(str, prompt)))]).split()
    for prompt, line in zip(prompts, produced):
        expected, margins = greedy_with_margin(config, tensors, prompt, 8)
        sure = next((i for i, margin in enumerate(margins) if margin < 1e-3), len(expected))
        assert [int(word) for word in line.split(",")][:sure] == expected[:sure] and sure > 2
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:70].tolist(), "want": [3, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[70:71].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[:2].tolist(), "want": [1]}], "end": ["a"]}]
    out = run("trace_run", "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "80",
              input="".join(json.dumps(step) + "\n" for step in steps))
    assert [line for line in out.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    for step, places in ((0, [3, 69]), (1, [70]), (2, [1])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(places), config["vocab"])
        assert cases.relative_error(got, want[places]).max() <= cases.LIMITS["float32"]

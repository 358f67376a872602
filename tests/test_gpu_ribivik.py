"""Ribivik in the framework against the plain restatement in float64: each mechanism alone in one-layer models, whole
models in portions of every kind, mixed batches, reused pages and slots, far keys and old state, and generation through
the serving engine."""
import numpy as np
import pytest

import ribivik_cases as cases
import stack_cases
from oracle import ribivik as oracle_ribivik

pytestmark = pytest.mark.gpu

TYPES = ("float32", "bfloat16")


def run_layers(config, tensors, device, dtype, portions, seed=3):
    """Residual stream behind the last layer, framework and restatement."""
    tokens = np.random.default_rng(seed).integers(0, config["vocab"], size=sum(portions)).astype(np.uint32)
    want, model = [], cases.oracle_model(config, tensors)
    model.forward(tokens, model.new_state(), want)
    got = stack_cases.residual_in_portions(
        lambda pages, slots: cases.product_model(config, tensors, device, dtype, pages, slots), device, tokens, portions)
    return got, want[-1]


def check_layers(config, seed, device, dtype, portions, change=None, exact=5e-6):
    """bf16: single tokens whose sublayer output nearly cancels get it back amplified by the norm behind it, so the bound on
    the typical token is the sharp one."""
    tensors = cases.random_tensors(config, seed)
    if change is not None:
        change(tensors)
    got, want = run_layers(config, tensors, device, dtype, portions)
    error = cases.relative_error(got, want)
    assert error.max() <= {"float32": exact, "bfloat16": 6e-2}[dtype], (int(error.argmax()), float(error.max()))
    assert np.median(error) <= {"float32": exact, "bfloat16": 1e-2}[dtype], float(np.median(error))


# ------------------------------------------------------------------------------------------------ mechanisms alone

LATENT_SHAPES = [   # heads, dim, rot_dim, vdim, q_rank, kv_rank
    (3, 24, 8, 16, 32, 40),            # sizes below one tensor-core chunk
    (8, 64, 64, 64, 64, 128),
    (16, 128, 64, 128, 96, 512),       # two key chunks and one shared, the widest latent
    (20, 48, 16, 40, 40, 192),         # more heads than one block of columns, an odd number of latent chunks
    (70, 16, 32, 24, 24, 64),          # several blocks of 64 heads
    (40, 32, 128, 32, 56, 448),        # a rotated part of two chunks
    (2, 192, 64, 128, 48, 96),
    (3, 200, 64, 72, 32, 64),          # keys beyond the prompt kernel
    (2, 64, 32, 136, 32, 64),          # values beyond it
    (2, 32, 16, 24, 32, 576),          # latents beyond the decode kernel
    (2, 20, 12, 10, 9, 22),            # no 16-byte rows anywhere
    (1, 8, 2, 8, 8, 8),
]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", LATENT_SHAPES, ids=lambda shape: "x".join(map(str, shape)))
def test_latent_attention_layer(device, dtype, shape):
    config = cases.config_of([cases.latent_layer(*shape, ff=0)])
    check_layers(config, 11, device, dtype, [75, 2, 1, 50, 1, 1, 90])


@pytest.mark.parametrize("dtype", TYPES)
def test_rotation_and_scale_alone(device, dtype):
    """Only the rotated part of the scores is left, with a scale that makes them sharp."""
    config = cases.config_of([cases.latent_layer(4, 16, 32, 32, 40, 64, base=30.0, scale=0.6, ff=0)])

    def only_rotated(tensors):
        tensors["l0.mix.uk"][:] = 0.0
    check_layers(config, 12, device, dtype, [60, 1, 5, 70, 1], change=only_rotated, exact=3e-5)


STATE_SHAPES = [    # heads, vdim, state, groups, norm_groups, conv
    (6, 8, 16, 3, 2, 3),
    (4, 64, 128, 1, 1, 4),
    (8, 64, 64, 2, 8, 4),
    (2, 128, 256, 2, 1, 4),
    (3, 48, 80, 1, 3, 4),
    (5, 40, 24, 5, 4, 2),
    (2, 16, 512, 1, 1, 4),
    (1, 96, 8, 1, 1, 1),
    (3, 10, 7, 1, 5, 4),               # no 16-byte rows anywhere
    (4, 20, 36, 2, 1, 7),
    (2, 8, 16, 1, 1, 24),              # a history longer than a tile of the convolution
]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", STATE_SHAPES, ids=lambda shape: "x".join(map(str, shape)))
def test_state_space_layer(device, dtype, shape):
    config = cases.config_of([cases.mamba_layer(*shape)])
    check_layers(config, 13, device, dtype, [70, 2, 1, 16, 1, 5, 133])


@pytest.mark.parametrize("shape", STATE_SHAPES[:5] + [(4, 64, 96, 2, 1, 4), (2, 24, 200, 1, 1, 4)],
                         ids=lambda shape: "x".join(map(str, shape)))
def test_state_space_prompt_kernels_agree(device, library_option, shape):
    """Chunks on the tensor cores and the token-by-token kernel on the same bf16 inputs: both keep the recurrence in 32
    bits, so they differ by rounding of the bf16 output only.  Decays from next to nothing to next to everything."""
    config = cases.config_of([cases.mamba_layer(*shape)])
    tensors = cases.random_tensors(config, 83)
    tensors["l0.mix.A_log"][:] = np.linspace(-6.0, 3.0, shape[0])
    results = []
    for forced in (0, 1):
        library_option("state_space_prompt", forced)
        results.append(run_layers(config, tensors, device, "bfloat16", [200, 33, 2, 16, 64, 3])[0])
    assert cases.relative_error(results[1], results[0]).max() < 4e-3


def test_latent_attention_kernels_agree(device, library_option):
    """Latents on the tensor cores, keys and values formed from them, and the plain kernel on the same inputs."""
    config = cases.config_of([cases.latent_layer(24, 64, 32, 48, 64, 256, scale=0.3, ff=0)])
    tensors = cases.random_tensors(config, 23)
    results = []
    for forced in (0, 1):
        library_option("stack_attention", forced)
        results.append(run_layers(config, tensors, device, "bfloat16", [130, 1, 70, 2, 1, 150, 1])[0])
    assert cases.relative_error(results[0], results[1]).max() < 1e-2


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("width,ff", [(48, 40), (256, 72), (64, 1000), (50, 30), (96, 9), (8448, 16)])
def test_feed_forward_and_its_norms(device, dtype, width, ff):
    """The mixer's output projection is zero: only the feed-forward with the norms before and after it is left."""
    config = cases.config_of([cases.mamba_layer(1, 16, 16, 1, 1, 2, ff=ff)], width=width)

    def only_feed_forward(tensors):
        tensors["l0.mix.o"][:] = 0.0
    check_layers(config, 17, device, dtype, [9, 2, 1], change=only_feed_forward)


@pytest.mark.parametrize("dtype", TYPES)
def test_small_outputs_are_normed_with_eps(device, dtype):
    """Sublayer outputs around sqrt(eps): eps inside the root decides how much of them enters the stream."""
    config = cases.config_of([cases.latent_layer(ff=24), cases.mamba_layer(ff=24)], eps=0.05)

    def shrink(tensors):
        for name in ("l0.mix.o", "l0.mlp.down", "l1.mix.o", "l1.mlp.down"):
            tensors[name] = cases.bf16_values(tensors[name] * 0.2)
    check_layers(config, 19, device, dtype, [20, 2, 1], change=shrink)


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
    cases.assert_logits(got, want, dtype)


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
        cases.assert_logits(np.concatenate(got[index]), want[index], dtype)


@pytest.mark.parametrize("dtype", TYPES)
def test_selected_places_only(device, dtype, mixed_case):
    config, tensors, tokens, want = mixed_case
    with cases.engine_of(config, tensors, device, dtype) as engine:
        assert engine.forced_step([(1, tokens[:40], [])], config["vocab"]).shape == (0, config["vocab"])
        places = [0, 1, 7, 8, 90, 109]
        got = engine.forced_step([(1, tokens[40:], places)], config["vocab"])
    cases.assert_logits(got, want[[40 + place for place in places]], dtype)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("sizes", [
    dict(vocab=101, width=40, eps=1e-6, softcap=0.0),
    dict(vocab=640 + 8, width=72, eps=1e-3, softcap=1.0),
    dict(vocab=33, width=30, eps=1e-5, softcap=50.0),        # width without 16-byte rows
    dict(vocab=256, width=128, eps=1e-5, softcap=5.0),       # shapes the tensor-core GEMMs take
], ids=lambda sizes: f"{sizes['vocab']}-{sizes['width']}-{sizes['softcap']}")
def test_other_sizes(device, dtype, sizes):
    layers = [cases.mamba_layer(5, 8, 40, 1, 5, 4, ff=24), cases.latent_layer(9, 24, 8, 40, 16, 136, base=77.0, scale=0.3, ff=0),
              cases.mamba_layer(4, 64, 128, 4, 2, 4, ff=136), cases.latent_layer(2, 8, 16, 8, 128, 64, ff=8),
              cases.latent_layer(3, 72, 8, 64, 8, 136, base=77.0, kv_from=1)]
    config = cases.config_of(layers, **sizes)
    tensors = cases.random_tensors(config, 41)
    tokens = np.random.default_rng(43).integers(0, config["vocab"], size=60)
    with cases.engine_of(config, tensors, device, dtype) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, [29, 2, 1, 12, 1, 15])
    cases.assert_logits(got, expected_logits(config, tensors, tokens), dtype)


@pytest.mark.parametrize("dtype", TYPES)
def test_long_decoding(device, dtype, mixed_case):
    config, tensors, _, _ = mixed_case
    tokens = np.random.default_rng(47).integers(0, config["vocab"], size=420)
    want = expected_logits(config, tensors, tokens)
    with cases.engine_of(config, tensors, device, dtype) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, [20] + [1] * 400)
    cases.assert_logits(got, want, dtype)


# ------------------------------------------------------------------------------------------------ keys that stand out

def standout_model(heads=4, kv_rank=64):
    """One layer in which the unrotated query of token 0 is the key of token 1 in every head, with a scale that lets one
    token 1 outweigh hundreds of others."""
    config = cases.config_of([cases.latent_layer(heads, 64, 16, 32, 32, kv_rank, base=1e6, scale=0.35, ff=0)], vocab=120,
                             width=128, softcap=20.0)
    tensors = cases.random_tensors(config, 53)
    eps = config["norm"]["eps"]
    asks, stands = (oracle_ribivik.shifted_norm(tensors["embed"][token], tensors["l0.norm1"], eps) for token in (0, 1))
    latent = oracle_ribivik.rms_norm((tensors["l0.mix.dkv"] @ stands)[:kv_rank], tensors["l0.mix.dkv.norm"], eps)
    keys = (tensors["l0.mix.uk"] @ latent).reshape(heads, 64)
    wanted = np.concatenate([keys, np.zeros((heads, 16))], axis=1).reshape(-1)
    compressed = oracle_ribivik.rms_norm(tensors["l0.mix.dq"] @ asks, tensors["l0.mix.dq.norm"], eps)
    weight = tensors["l0.mix.uq"]
    tensors["l0.mix.uq"] = cases.bf16_values(
        weight + np.outer(wanted - weight @ compressed, compressed) / (compressed @ compressed))
    return config, tensors


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("how", ["prompt", "decoded", "pair"])
@pytest.mark.parametrize("key,query", [(0, 1), (0, 15), (0, 16), (15, 16), (15, 63), (16, 64), (63, 64), (63, 128),
                                       (64, 127), (64, 191), (1, 255), (0, 256), (127, 300), (128, 301), (255, 320),
                                       (0, 333), (332, 333)])
def test_far_keys_and_page_borders(device, dtype, how, key, query):
    """Token 1 stands at `key` only, token 0 asks at the end: one place of the key axis decides the answer.  The restatement
    itself proves that the case is sharp."""
    config, tensors = standout_model()
    tokens = np.random.default_rng(59).integers(2, config["vocab"], size=query + 1)
    tokens[query] = 0
    other = tokens.copy()                         # the same with an ordinary token at `key`
    tokens[key] = 1
    want = expected_logits(config, tensors, tokens)[-1:]
    moved = cases.relative_error(expected_logits(config, tensors, other)[-1:], want).max()
    assert moved > 2 * cases.SHARP[dtype]
    portions = {"prompt": [query + 1], "decoded": [query, 1], "pair": [query - 1, 2] if query > 1 else [query + 1]}[how]
    with cases.engine_of(config, tensors, device, dtype) as engine:
        got = cases.feed(engine, config["vocab"], 1, tokens, portions)[-1:]
    cases.assert_logits(got, want, dtype)


@pytest.mark.parametrize("splits", [700, 2100])
def test_splits_of_long_contexts(device, splits):
    """Contexts long enough for the decode kernel to split them: the standing-out key in every part of the range."""
    config, tensors = standout_model(heads=18, kv_rank=128)
    rng = np.random.default_rng(61)
    base = rng.integers(2, config["vocab"], size=splits)
    with cases.engine_of(config, tensors, device, "bfloat16", num_pages=600, slots=4, sequence_tokens=2304,
                         prefill_tokens=512) as engine:
        for number, key in enumerate((0, 1, 63, 64, 130, splits // 2, splits - 65, splits - 2)):
            tokens = base.copy()
            tokens[key], tokens[-1] = 1, 0
            engine.forced_step([(number, tokens[:-1], [])], config["vocab"])
            got = engine.forced_step([(number, tokens[-1:], [0])], config["vocab"])
            engine.end_forced(number)
            # only the last token matters for one layer: the restatement attends from it alone
            model = cases.oracle_model(config, tensors)
            want = last_token_logits(model, tokens)
            assert cases.relative_error(got, want[None]).max() <= cases.SHARP["bfloat16"], key


def last_token_logits(model, tokens):
    """One-layer latent attention, the last token's logits only (the others' queries do not enter them)."""
    config, tensors, eps = model.config, model.tensors, model.config["norm"]["eps"]
    sizes, mixer = config["layers"][0]["mixer"], model._mixer_tensors(0)
    x = tensors["embed"][np.asarray(tokens)]
    h = oracle_ribivik.shifted_norm(x, tensors["l0.norm1"], eps)
    rot = sizes["rot"]
    latent, key = oracle_ribivik.latent_entries(h[:-1], mixer, sizes["kv_rank"], np.arange(len(tokens) - 1), rot["base"],
                                                rot["dims"], eps)
    update = oracle_ribivik.latent_attention(h[-1:], mixer, sizes, eps, np.array([len(tokens) - 1]), [latent, key])
    x = x[-1:] + oracle_ribivik.shifted_norm(update, tensors["l0.norm1b"], eps)
    final = oracle_ribivik.shifted_norm(x, tensors["final.norm"], eps)
    return oracle_ribivik.softcap(oracle_ribivik.linear(final, tensors["head"]), config["logit_softcap"])[0]


@pytest.mark.parametrize("dtype", TYPES)
def test_growing_scores_move_the_reference(device, dtype):
    """Scores that climb along the sequence by far more than a factor of 2^8 from one stage of keys to the next: earlier
    weights shrink to almost nothing every time."""
    config, tensors = standout_model()
    tokens = np.random.default_rng(67).integers(2, config["vocab"], size=400)
    ladder = [5, 70, 140, 210, 290, 398]
    # tokens 3 .. 8 lie between token 2 and token 1 in embedding space, ever closer to token 1
    for step, place in enumerate(ladder):
        mix = (step + 1) / len(ladder)
        tensors["embed"][3 + step] = cases.bf16_values((1 - mix) * tensors["embed"][2] + mix * tensors["embed"][1])
    tokens[(tokens >= 3) & (tokens < 9)] = 50
    for step, place in enumerate(ladder):
        tokens[place] = 3 + step
    tokens[-1] = 0
    want = expected_logits(config, tensors, tokens)[-1:]
    for portions in ([400], [399, 1], [398, 2]):
        with cases.engine_of(config, tensors, device, dtype) as engine:
            got = cases.feed(engine, config["vocab"], 1, tokens, portions)[-1:]
        cases.assert_logits(got, want, dtype)


@pytest.mark.parametrize("dtype", TYPES)
def test_state_reaches_far_back(device, dtype):
    """Decays close to one and a first token that outweighs the rest: what it wrote is still read 200 tokens on, across
    portions and decoding."""
    config = cases.config_of([cases.mamba_layer(4, 32, 32, 1, 1, 2)], vocab=60, width=64, softcap=0.0)
    tensors = cases.random_tensors(config, 71)
    tensors["l0.mix.A_log"][:] = -12.0
    tensors["l0.mix.D"][:] = 0.0
    tensors["embed"][1:] = tensors["embed"][1:] * 0.5
    tokens = np.random.default_rng(73).integers(2, config["vocab"], size=200)
    tokens[0] = 0
    tensors["l0.mix.dt_bias"][:] = -4.0
    first = oracle_ribivik.shifted_norm(tensors["embed"][0], tensors["l0.norm1"], 1e-4)
    raw = tensors["l0.mix.in"]
    raw[-4:] = 0.0                                                     # step sizes: large for the first token only
    raw[-4:] = cases.bf16_values(np.tile(first * 12.0 / (first @ first), (4, 1)))
    other = tokens.copy()
    other[0] = 1
    want = expected_logits(config, tensors, tokens)
    moved = cases.relative_error(expected_logits(config, tensors, other)[-1:], want[-1:]).max()
    assert moved > 20 * cases.SHARP["float32"]
    for portions in ([200], [3, 64, 1, 1, 100, 1, 30], [150] + [1] * 50):
        with cases.engine_of(config, tensors, device, dtype) as engine:
            got = cases.feed(engine, config["vocab"], 1, tokens, portions)
        cases.assert_logits(got, want, dtype)


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
    """A prompt whose beginning was served before takes its pages from the index and its recurrent states from the
    checkpoint."""
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
    for dtype in TYPES:
        out = run("trace_run", "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "80",
                  input="".join(json.dumps(step) + "\n" for step in steps))
        assert [line for line in out.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
        for step, places in ((0, [3, 69]), (1, [70]), (2, [1])):
            got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(places), config["vocab"])
            assert cases.relative_error(got, want[places]).max() <= cases.SHARP[dtype]


@pytest.mark.parametrize("portions", [[180], [90, 2, 1, 1, 60, 26], [179, 1]], ids=["whole", "mixed", "decoded"])
def test_pages_that_hold_not_a_number(device, portions):
    """What a page held before it was handed out reaches no result: caches full of NaN patterns around the sequence."""
    import torch
    config = cases.config_of([cases.latent_layer(6, 64, 32, 32, 48, 96, ff=0), cases.latent_layer(2, kv_rank=40, ff=0)])
    tensors = cases.random_tensors(config, 89)
    tokens = np.random.default_rng(91).integers(0, config["vocab"], size=180).astype(np.uint32)
    want, model = [], cases.oracle_model(config, tensors)
    model.forward(tokens, model.new_state(), want)
    for dtype in TYPES:
        def poisoned(pages, slots):
            made = cases.product_model(config, tensors, device, dtype, pages, slots)
            for pair in made.caches:
                for cache in pair:
                    cache.fill_(float("nan"))
            torch.cuda.current_stream().synchronize()
            return made
        got = stack_cases.residual_in_portions(poisoned, device, tokens, portions)
        assert cases.relative_error(got, want[-1]).max() <= {"float32": 1e-5, "bfloat16": 6e-2}[dtype]

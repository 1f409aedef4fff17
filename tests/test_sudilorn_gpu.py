"""The Sudilorn design in the engine against the plain implementation (``plain/sudilorn.py``), on tiny models of five different
make-ups: whole prompts, decoding token by token behind a prompt, portions down to two tokens, mixed batches on pools so
small that pages and state slots are used again, long decoding, and greedy generation through ``LLM.generate``; in 32-bit
(equal to the plain implementation's float64 up to float32 rounding) and in bfloat16 (weights rounded once, compared on the
same rounded weights)."""

import numpy as np
import pytest

import replay_util as ru
from plain import sudilorn as plain
from tiny_sudilorn import CALM, TINY, make_model_dir

pytestmark = pytest.mark.gpu

# Largest difference of a position's logits over their spread there.
F32_TOLERANCE = 1e-3
# bfloat16: a router's choice is a step function, and where two experts lie within rounding of each other bfloat16 may take
# the other one.  Models whose routers decide far from any tie are held to the plain implementation at every position; the
# others on most positions, and to the engine's own logits for each request alone and whole on most (what the schedule, the
# pages and the slots could change).
# What bfloat16's rounding of activations alone does to the plain implementation, a few times over: the peaked heads of Z4
# amplify it most.
BF16_TOLERANCE = {"Z1": 0.25, "Z2": 0.25, "Z3": 0.25, "Z4": 0.5, "Z5": 0.1}
BF16_SHARE, BF16_SCHEDULE_TOLERANCE, BF16_SCHEDULE_SHARE = 0.75, 0.15, 0.80


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("sudilorn")
    return {(name, dtype): make_model_dir(root, name, dtype) for name in TINY for dtype in ("float32", "bfloat16")}


def requests_for(name, lengths, seed=0):
    vocab = TINY[name][0]["vocab"]
    rng = np.random.default_rng(seed)
    return {f"q{i}": rng.integers(0, vocab, size=n).tolist() for i, n in enumerate(lengths)}


_wanted = {}


def oracle(folder, requests):
    """The plain logits of every request, each computed once per run."""
    loaded = None
    for ids in requests.values():
        key = (folder, tuple(ids))
        if key not in _wanted:
            loaded = loaded or plain.load_model_dir(folder, np.float64)
            _wanted[key] = plain.forward_logits(*loaded, ids)
    return {rid: _wanted[folder, tuple(ids)] for rid, ids in requests.items()}


def relative_errors(got, want):
    return np.abs(got - want).max(axis=1) / np.maximum(want.std(axis=1), 1e-3)


def check(name, dtype, folders, requests, steps, max_requests=4, max_tokens=None):
    folder = folders[name, dtype]
    want = oracle(folder, requests)
    got, runner = ru.run_in_process(folder, dtype, steps, max_tokens or ru.max_live_tokens(steps), TINY[name][2], max_requests)
    bound = F32_TOLERANCE if dtype == "float32" else BF16_TOLERANCE[name]
    errors = {rid: relative_errors(got[rid], want[rid]) for rid in requests}
    if dtype == "float32" or name in CALM:
        for rid, err in errors.items():
            assert err.max() < bound, f"{name} request {rid}: first wrong token {int(np.argmax(err >= bound))}, worst error {err.max():.2e}"
    else:
        err = np.concatenate(list(errors.values()))
        assert np.mean(err < bound) >= BF16_SHARE, f"{name}: {np.mean(err < bound):.2f} of the positions"
        alone = ru.whole(requests)
        if steps != alone:
            base, _ = ru.run_in_process(folder, dtype, alone, ru.max_live_tokens(alone), TINY[name][2], 4)
            diff = np.concatenate([relative_errors(got[rid], base[rid]) for rid in requests])
            share = np.mean(diff < BF16_SCHEDULE_TOLERANCE)
            assert share >= BF16_SCHEDULE_SHARE, f"{name}: {share:.3f} of the positions equal the whole prompt's, worst {diff.max():.2e}"
    runner.cache.check(runner.live.values())
    assert not runner.live and all(n == 0 for n in runner.cache.pages_in_use())
    return runner


LENGTHS = {"Z1": [1, 2, 67, 150], "Z2": [3, 40, 300], "Z3": [5, 200, 31], "Z4": [1, 77, 200], "Z5": [2, 141]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY))
def test_whole_prompts(folders, name, dtype):
    """Prompts of one and two tokens among them (windows and convolutions that reach before the start, the first token's own
    key), and prompts of several windows and chunks."""
    requests = requests_for(name, LENGTHS[name])
    check(name, dtype, folders, requests, ru.whole(requests))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY))
def test_prompt_then_token_by_token(folders, name, dtype):
    """The last 48 tokens one by one: keys that leave the window while decoding, kept tokens, memories and the convolutions'
    inputs carried from the prompt's kernels into single tokens."""
    requests = requests_for(name, [l for l in LENGTHS[name] if l > 2], seed=1)
    check(name, dtype, folders, requests, ru.prefill_then_decode(requests, tail=48))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY))
def test_portions_of_many_sizes(folders, name, dtype):
    """Cuts in the middle of pages, windows, chunks and the convolutions' windows: portions of 2, 3, 1, 17, 5, 64 tokens, of two
    tokens only, and of sizes on both sides of the cut between walking and chunking."""
    requests = requests_for(name, [max(LENGTHS[name]), 37], seed=2)
    check(name, dtype, folders, requests, ru.portions(requests, [2, 3, 1, 17, 5, 64]))
    check(name, dtype, folders, requests, ru.portions(requests, [15, 16, 65, 2]))
    short = requests_for(name, [29], seed=8)
    check(name, dtype, folders, short, ru.portions(short, [2]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY))
def test_mixed_batches_reuse_pages_and_slots(folders, name, dtype):
    """Seven requests through three state slots and a pool that holds just the live ones: portions beside single tokens,
    unequal lengths, every slot and page used again by a later request; each request's logits equal those it gets
    alone (the plain implementation sees one request at a time)."""
    requests = requests_for(name, [90, 7, 130, 33, 2, 61, 48], seed=3)
    steps = ru.mixed(requests, seed=5, max_live=3, decode_tail=9)
    runner = check(name, dtype, folders, requests, steps, max_requests=3)
    assert runner.steps == len(steps)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["Z2", "Z4"])
def test_long_portions_beside_single_tokens(folders, name, dtype):
    """Runs that go in chunks, runs that are walked and single tokens of others in one step."""
    requests = requests_for(name, [40, 230, 150, 25], seed=6)
    cuts = {"q0": [30] + [1] * 10, "q1": [100, 2, 128], "q2": [1, 145, 4], "q3": [20, 3, 1, 1]}
    at, steps, k = {r: 0 for r in requests}, [], 0
    while any(at[r] < len(requests[r]) for r in requests):
        entries, end = [], []
        for r in requests:
            if k < len(cuts[r]):
                n = cuts[r][k]
                entries.append({"id": r, "tokens": requests[r][at[r]:at[r] + n], "want": list(range(n))})
                at[r] += n
                if at[r] == len(requests[r]):
                    end.append(r)
        steps.append({"step": k, "entries": entries, "end": end})
        k += 1
    check(name, dtype, folders, requests, steps)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["Z1", "Z2"])
def test_long_decoding(folders, name, dtype):
    """260 tokens one by one behind a prompt of three: steps replayed from captured graphs, memories that have been decayed
    and written hundreds of times, windows that have let go of most pages while the kept tokens' stay."""
    requests = requests_for(name, [263], seed=4)
    runner = check(name, dtype, folders, requests, ru.prefill_then_decode(requests, tail=260))
    assert runner.graph_replays > 200


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["Z1", "Z2", "Z3"])
def test_greedy_generation_through_the_scheduler(folders, name, dtype):
    """``LLM.generate``: the engine's own entry point, scheduler (portions of 16 tokens, three requests on two seats; decode
    steps packed before their tokens are known) and sampler; 32-bit reproduces the plain implementation's tokens, bfloat16
    (where no router is near a tie) chooses tokens whose plain logits lie within rounding of the largest."""
    from qwen25vl_lite import LLM, SamplingParams

    folder = folders[name, dtype]
    prompts = list(requests_for(name, [5, 41, 18], seed=7).values())
    llm = LLM(folder, dtype=dtype, num_blocks=48, block_size=TINY[name][2], max_num_seqs=2, max_num_batched_tokens=16)
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    cfg, w = plain.load_model_dir(folder, np.float64)
    for p, o in zip(prompts, outs):
        assert len(o.output_token_ids) == 12
        if dtype == "float32":
            assert o.output_token_ids == plain.greedy_generate(cfg, w, p, 12)
        elif name in CALM:
            spread = float(plain.forward_logits(cfg, w, list(p) + list(o.output_token_ids)).std(axis=1).mean())
            assert max(plain.generation_margins(cfg, w, p, o.output_token_ids)) < 2 * BF16_TOLERANCE[name] * spread
    llm.runner.cache.check(llm.runner.live.values())


def test_generation_of_many_requests_pads_its_batches(folders):
    """Eleven requests decode together (a captured step of 16 rows, five of them padding that share a page and a slot): their
    tokens are those each gets alone."""
    from qwen25vl_lite import LLM, SamplingParams

    folder = folders["Z2", "float32"]
    prompts = list(requests_for("Z2", [4 + 3 * i for i in range(11)], seed=9).values())
    make = lambda seats: LLM(folder, dtype="float32", num_blocks=200, block_size=8, max_num_seqs=seats, max_num_batched_tokens=256)
    together, alone = make(16), make(1)
    params = SamplingParams(max_tokens=15, ignore_eos=True)
    assert [o.output_token_ids for o in together.generate(prompts, params)] == [o.output_token_ids for o in alone.generate(prompts, params)]
    assert together.runner.graph_replays > 0

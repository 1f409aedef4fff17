"""The Mezinex design in the engine against the plain implementation (``plain/mezinex.py``), on tiny models of five
different make-ups: whole prompts, decoding token by token behind a prompt, portions down to two tokens, mixed batches
on pools so small that pages and state slots are used again, long decoding, and greedy generation through
``LLM.generate``; in 32-bit (equal to the plain implementation's float64 up to float32 rounding) and in bfloat16
(weights rounded once, compared on the same rounded weights)."""

import numpy as np
import pytest

import replay_util as ru
from plain import mezinex as plain
from tiny_mezinex import TINY, make_model_dir

pytestmark = pytest.mark.gpu

# Largest difference of a position's logits over their spread there.  The design has no router and no other step
# function, so bfloat16 is held to the plain implementation at every position too.
F32_TOLERANCE = 5e-4
BF16_TOLERANCE = 0.25


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("mezinex")
    return {(name, dtype): make_model_dir(root, name, dtype) for name in TINY for dtype in ("float32", "bfloat16")}


def requests_for(name, lengths, seed=0):
    vocab = TINY[name][0]["vocab"]
    rng = np.random.default_rng(seed)
    return {f"q{i}": rng.integers(0, vocab, size=n).tolist() for i, n in enumerate(lengths)}


def oracle(folder, requests):
    cfg, w = plain.load_model_dir(folder, np.float64)
    return {rid: plain.forward_logits(cfg, w, ids) for rid, ids in requests.items()}


def relative_errors(got, want):
    return np.abs(got - want).max(axis=1) / np.maximum(want.std(axis=1), 1e-3)


def check(name, dtype, folders, requests, steps, max_requests=4, max_tokens=None):
    folder = folders[name, dtype]
    want = oracle(folder, requests)
    got, runner = ru.run_in_process(folder, dtype, steps, max_tokens or ru.max_live_tokens(steps), TINY[name][2], max_requests)
    bound = F32_TOLERANCE if dtype == "float32" else BF16_TOLERANCE
    for rid in requests:
        assert got[rid].shape == want[rid].shape
        err = relative_errors(got[rid], want[rid])
        assert err.max() < bound, f"{name} request {rid}: first wrong token {int(np.argmax(err >= bound))}, worst error {err.max():.2e}"
    runner.cache.check(runner.live.values())
    assert not runner.live and all(n == 0 for n in runner.cache.pages_in_use())
    return runner


LENGTHS = {"Z1": [1, 2, 67, 150], "Z2": [3, 40, 300], "Z3": [5, 260, 31], "Z4": [1, 77, 200], "Z5": [2, 141]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY))
def test_whole_prompts(folders, name, dtype):
    """Prompts of one and two tokens among them (the pair of a first token, windows of the convolutions that reach before
    the start), and prompts of several chunks of the state space's walk."""
    requests = requests_for(name, LENGTHS[name])
    check(name, dtype, folders, requests, ru.whole(requests))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY))
def test_prompt_then_token_by_token(folders, name, dtype):
    """The last 48 tokens one by one: latents across page borders, every state carried from the prompt's kernels into single
    tokens, the previous token of every pair, every pass of a looped stretch with its own pages and slots."""
    requests = requests_for(name, [l for l in LENGTHS[name] if l > 2], seed=1)
    check(name, dtype, folders, requests, ru.prefill_then_decode(requests, tail=48))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY))
def test_portions_of_many_sizes(folders, name, dtype):
    """Cuts in the middle of pages, of chunks and of the convolutions' windows: portions of 2, 3, 1, 17, 5, 64 tokens, of two
    tokens only, and of sizes on both sides of the cut between walking and chunking."""
    requests = requests_for(name, [max(LENGTHS[name]), 37], seed=2)
    check(name, dtype, folders, requests, ru.portions(requests, [2, 3, 1, 17, 5, 64]))
    check(name, dtype, folders, requests, ru.portions(requests, [127, 2, 128]))
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
def test_long_portions_beside_single_tokens(folders, dtype):
    """Runs that are cut into chunks and runs that are walked, in one step with single tokens of others."""
    requests = requests_for("Z1", [40, 330, 210, 25], seed=6)
    cuts = {"q0": [30] + [1] * 10, "q1": [150, 2, 178], "q2": [1, 205, 4], "q3": [20, 3, 1, 1]}
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
    check("Z1", dtype, folders, requests, steps)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["Z1", "Z2"])
def test_long_decoding(folders, name, dtype):
    """260 tokens one by one behind a prompt of three: steps replayed from captured graphs, states that have been decayed
    hundreds of times, latents over many pages, the pair's previous token read on the device."""
    requests = requests_for(name, [263], seed=4)
    runner = check(name, dtype, folders, requests, ru.prefill_then_decode(requests, tail=260))
    assert runner.graph_replays > 200


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["Z1", "Z3", "Z5"])
def test_greedy_generation_through_the_scheduler(folders, name, dtype):
    """``LLM.generate``: the engine's own entry point, scheduler (portions of 16 tokens, three requests on two seats; decode
    steps packed before their tokens are known) and sampler; 32-bit reproduces the plain implementation's tokens,
    bfloat16 chooses tokens whose plain logits lie within rounding of the largest."""
    from qwen25vl_lite import LLM, SamplingParams

    folder = folders[name, dtype]
    prompts = list(requests_for(name, [5, 41, 18], seed=7).values())
    llm = LLM(folder, dtype=dtype, num_blocks=48, block_size=TINY[name][2], max_num_seqs=2, max_num_batched_tokens=16)
    outs = llm.generate(prompts, SamplingParams(max_tokens=20, ignore_eos=True))
    cfg, w = plain.load_model_dir(folder, np.float64)
    for p, o in zip(prompts, outs):
        assert len(o.output_token_ids) == 20
        if dtype == "float32":
            assert o.output_token_ids == plain.greedy_generate(cfg, w, p, 20)
        else:
            spread = float(plain.forward_logits(cfg, w, list(p) + list(o.output_token_ids)).std(axis=1).mean())
            assert max(plain.generation_margins(cfg, w, p, o.output_token_ids)) < 2 * BF16_TOLERANCE * spread
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

"""The kernels of the Mezinex design's mechanisms, each alone against plain float64 arithmetic, with inputs made so that a
fault shows: rows of the stream of very different sizes under a mixing matrix that is far from symmetric; pair products
beyond 32 bits, first tokens and tokens behind a cut; convolutions over portions shorter than their window; heads that
never forget beside heads that forget at once, a single large step that only a far token reads; norm parts of very
different sizes; a far latent key that carries the whole weight among hundreds."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import mezinex as plain
from qwen25vl_lite.engine.runner import HostStep, KVStep
from qwen25vl_lite.ops import attention as attention_ops
from qwen25vl_lite.ops import kernels, state_space

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)
f32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)
npy = lambda t: t.detach().double().cpu().numpy()


# ---- the stream of several rows ------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams,width", [(1, 96), (2, 100), (3, 96), (4, 2048), (5, 64), (7, 50), (16, 36)])
def test_stream_is_written_and_read(dtype, streams, width):
    """The pending result enters all rows at once from the old ones, then the norm of the weighted sum of the new rows; with
    nothing pending; on chosen rows, which leave the stream as it is; the plain sum."""
    g = torch.Generator(device=DEV).manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    n = 9
    x = rnd(n, streams, width) * torch.tensor([10.0 ** (s % 3 - 1) for s in range(streams)], device=DEV)[:, None]
    y, mix, ow, iw, w = rnd(n, width).to(dtype), rnd(streams, streams), rnd(streams), rnd(streams), rnd(width) + 1.5
    new = plain.hyper_write(npy(x).transpose(1, 0, 2), npy(mix), npy(ow), npy(y))
    want = plain.rms_unit(plain.hyper_read(new, npy(iw)), 1e-5) * npy(w)
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    x1, out = x.clone(), torch.empty(n, width, dtype=dtype, device=DEV)
    kernels.hyper_norm(x1, y, mix, ow, iw, w, 1e-5, out)
    np.testing.assert_allclose(npy(x1).transpose(1, 0, 2), new, rtol=1e-5, atol=1e-4)
    np.testing.assert_allclose(npy(out), want, **tol)
    if streams > 1:
        turned = plain.hyper_write(npy(x).transpose(1, 0, 2), npy(mix).T, npy(ow), npy(y))
        assert np.abs(turned - new).max() > 0.1
    x2, some = x.clone(), torch.empty(3, width, dtype=dtype, device=DEV)
    kernels.hyper_norm(x2, y, mix, ow, None, w, 1e-5, some, i32([5, 0, 8]))
    assert torch.equal(x2, x)
    np.testing.assert_allclose(npy(some), (plain.rms_unit(new.sum(axis=0), 1e-5) * npy(w))[[5, 0, 8]], **tol)
    kernels.hyper_norm(x2, None, None, None, iw, w, 1e-5, out)
    assert torch.equal(x2, x)
    np.testing.assert_allclose(npy(out), plain.rms_unit(plain.hyper_read(npy(x).transpose(1, 0, 2), npy(iw)), 1e-5) * npy(w), **tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(601, 29, 13), (7, 900_000_007, 4_000_000_019), (1, 2, 3)])
def test_pairs_of_tokens_across_cuts_and_slots(dtype, buckets, mul_prev, mul_cur):
    """Three requests in turns of uneven portions through slots in another order than the batch; then one slot is used
    again by a new request, whose first token must not see the old one's last."""
    g = torch.Generator(device=DEV).manual_seed(2)
    vocab, width, streams = 50_000, 36, 3
    table = torch.randn(vocab, width, generator=g, device=DEV).to(dtype)
    pairs = torch.randn(buckets + 1, width, generator=g, device=DEV).to(dtype)
    last = torch.full((4,), 12345, dtype=torch.int32, device=DEV)
    rng = np.random.default_rng(2)
    ids = {r: rng.integers(0, vocab, size=40).tolist() for r in "abcd"}
    slots, at = {"a": 2, "b": 0, "c": 3, "d": 2}, dict.fromkeys("abcd", 0)
    for step in [dict(a=5, b=1, c=2), dict(c=1, a=1, b=1), dict(b=9, a=2), dict(a=32, c=1), dict(d=3, c=30), dict(d=1, b=1), dict(d=1)]:
        toks, seq, cu, start, slot = [], [], [0], [], []
        for i, (r, n) in enumerate(step.items()):
            toks += ids[r][at[r]:at[r] + n]
            seq += [i] * n
            cu.append(cu[-1] + n)
            start.append(at[r])
            slot.append(slots[r])
        x = torch.empty(len(toks), streams, width, device=DEV)
        kernels.hyper_embed(table, pairs, i32(toks), i32(seq), i32(cu), i32(start), i32(slot), last, x, buckets, mul_prev, mul_cur)
        for i, (r, n) in enumerate(step.items()):
            rows = plain.bigram_rows(ids[r][:at[r] + n], buckets, mul_prev, mul_cur)[at[r]:]
            want = table[ids[r][at[r]:at[r] + n]].float() + pairs[rows].float()
            for s in range(streams):
                assert torch.equal(x[cu[i]:cu[i + 1], s], want), f"request {r} from token {at[r]}"
            at[r] += n
    x = torch.empty(4, 1, width, device=DEV)                    # without a pair table
    kernels.hyper_embed(table, None, i32([3, 1, 2, 3]), i32([0, 0, 0, 0]), i32([0, 4]), i32([0]), i32([0]), None, x)
    assert torch.equal(x[:, 0], table[[3, 1, 2, 3]].float())


# ---- the state space -------------------------------------------------------------------------------------------------


def portions_of(total, sizes):
    out, k = [], 0
    while sum(out) < total:
        out.append(min(sizes[k % len(sizes)], total - sum(out)))
        k += 1
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(96, 4), (75, 3), (64, 1), (130, 2), (33, 7), (40, 16)])
@pytest.mark.parametrize("silu", [True, False])            # False: the result in float32
def test_convolution_over_portions(dtype, channels, taps, silu):
    """Two requests at once, one whole in long portions, one in portions shorter than the window; the history sits behind
    other state in the slots; what the slots hold elsewhere is left alone."""
    g = torch.Generator(device=DEV).manual_seed(3)
    total, off = 150, 17
    wide = torch.randn(2, total, channels + 11, generator=g, device=DEV).to(dtype)      # strided rows
    w, b = torch.randn(taps, channels, generator=g, device=DEV), torch.randn(channels, generator=g, device=DEV)
    state = torch.zeros(3, off + (taps - 1) * channels + 5, device=DEV)
    state[:, :off], state[:, off + (taps - 1) * channels:] = 7.0, 8.0
    cuts = [portions_of(total, [100, 1, 49]), portions_of(total, [1, 2, 3, 1, 5])]
    slots, at, got = [2, 0], [0, 0], [[], []]
    for k in range(max(len(c) for c in cuts)):
        live = [i for i in range(2) if k < len(cuts[i])]
        lens = [cuts[i][k] for i in live]
        x = torch.cat([wide[i, at[i]:at[i] + n] for i, n in zip(live, lens)])[:, 4:4 + channels]
        out = torch.empty(sum(lens), channels, dtype=dtype if silu else torch.float32, device=DEV)
        kernels.causal_conv(x, w, b, state, off, i32(np.cumsum([0] + lens)), i32([slots[i] for i in live]), out, len(live), max(lens), silu)
        for i, part in zip(live, torch.split(out, lens)):
            got[i].append(npy(part))
        for i, n in zip(live, lens):
            at[i] += n
    for i in range(2):
        want = plain.causal_conv(npy(wide[i, :, 4:4 + channels]), npy(w).T, npy(b))
        want = plain.silu(want) if silu else want
        np.testing.assert_allclose(np.concatenate(got[i]), want, **(dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)))
    assert (state[:, :off] == 7.0).all() and (state[:, off + (taps - 1) * channels:] == 8.0).all() and (state[1, off:-5] == 0).all()


def ssd_case(dtype, H, G, N, V, total, seed):
    """Rows [x | B | C], steps, and per-head constants: head 0 keeps everything (a decay of almost 1), head 1 forgets at
    once, the others are in between."""
    g = torch.Generator(device=DEV).manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    rows = (rnd(total, H * V + 2 * G * N) * 0.5).to(dtype)
    steps = rnd(total, H) - 2.0
    bias = rnd(H) * 0.3
    a_log = torch.linspace(-3.0, 1.0, H, device=DEV)
    a_log[0] = -15.0
    if H > 1:
        a_log[1] = 3.0
    return rows, steps, bias, a_log


def ssd_want(rows, steps, bias, a_log, H, G, N, V):
    T = rows.shape[0]
    x, b, c = np.split(npy(rows), [H * V, H * V + G * N], axis=-1)
    dt = plain.softplus(npy(steps) + npy(bias))
    return plain.state_space(x.reshape(T, H, V), b.reshape(T, G, N), c.reshape(T, G, N), dt, npy(a_log), np.zeros(H))


def run_ssd(rows, steps, bias, a_log, H, G, N, V, lens, starts, slots, state, tensor_cores=True):
    """One step over entries (their first rows in ``starts``); returns the outputs per entry.  ``tensor_cores`` False: the
    walk alone."""
    x = torch.cat([rows[s:s + n] for s, n in zip(starts, lens)])
    z = torch.cat([steps[s:s + n] for s, n in zip(starts, lens)]).contiguous()
    o = torch.empty(x.shape[0], H, V, device=DEV)
    mma = tensor_cores and kernels.state_space_mma_supports(x.dtype, H, G, N, V)
    work = {k: (i32(v) if len(v) else None) for k, v in state_space.plan(list(lens), mma).items()}
    ctx = SimpleNamespace(cu_q=i32(np.cumsum([0] + list(lens))), slot_ids=i32(slots), n_seqs=len(lens))
    state_space.run(work, ctx, x, H * V + G * N, H * V, 0, z, bias, a_log, state, o, H, G, N, V)
    return torch.split(o, list(lens))


SSD_SIZES = [(4, 2, 32, 16), (6, 3, 24, 20), (5, 5, 10, 14), (3, 1, 128, 64), (2, 1, 64, 64), (4, 1, 128, 128), (2, 2, 160, 40), (8, 1, 64, 32),
             (6, 2, 32, 56), (6, 3, 128, 40), (96, 4, 64, 64), (90, 1, 128, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,V", SSD_SIZES)
def test_state_space_whole_cut_and_decoded(dtype, H, G, N, V):
    """The same request whole, in portions from one token to several chunks, and token by token at its end: the walk, the
    chunked passes and single tokens give the plain result, and leave the same state."""
    total = 333 if H < 50 else 150
    rows, steps, bias, a_log = ssd_case(dtype, H, G, N, V, total, 5)
    want = ssd_want(rows, steps, bias, a_log, H, G, N, V)
    scale = np.abs(want).max(axis=(0, 2))[:, None]
    tol = 2e-5 if dtype == torch.float32 else 1e-4
    ends = []
    for sizes, cores in (([total], True), ([total], False), ([50, 1, 1, 2, 64, 65, 50, 100], True), ([130] * 2 + [1] * 73, True),
                         ([17, 127, 128, 61], True)):
        sizes = portions_of(total, sizes)
        state = torch.zeros(2, H * N * V + 9, device=DEV)
        at, got = 0, []
        for n in sizes:
            got.append(npy(run_ssd(rows, steps, bias, a_log, H, G, N, V, [n], [at], [1], state, cores)[0]))
            at += n
        # the inputs are the rounded ones on both sides and everything behind them is float32 (or carries 16 bits)
        assert (np.abs(np.concatenate(got) - want) / scale).max() < tol, f"portions {sizes}, tensor cores {cores}"
        assert (state[0] == 0).all() and (state[1, H * N * V:] == 0).all()
        ends.append(npy(state[1]))
    for e in ends[1:]:
        np.testing.assert_allclose(e, ends[0], rtol=tol, atol=tol * np.abs(ends[0]).max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,V", [(4, 2, 32, 16), (3, 1, 128, 64), (40, 1, 64, 64)])
def test_state_space_batches_of_unequal_entries(dtype, H, G, N, V):
    """Long runs, short runs and single tokens of different requests in one step equal each alone, bit for bit."""
    rows, steps, bias, a_log = ssd_case(dtype, H, G, N, V, 700, 6)
    lens, starts, slots = [1, 300, 40, 129, 2, 128], [0, 1, 301, 341, 470, 472], [5, 0, 3, 1, 4, 2]
    state = torch.randn(6, H * N * V, generator=torch.Generator(device=DEV).manual_seed(1), device=DEV)
    before = state.clone()
    together = run_ssd(rows, steps, bias, a_log, H, G, N, V, lens, starts, slots, state)
    for i, (n, s, slot) in enumerate(zip(lens, starts, slots)):
        own = before.clone()
        alone = run_ssd(rows, steps, bias, a_log, H, G, N, V, [n], [s], [slot], own)[0]
        assert torch.equal(alone, together[i]) and torch.equal(own[slot], state[slot])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("far", [63, 64, 127, 128, 400])
def test_a_far_token_reads_a_single_large_step(dtype, far):
    """Only the first token writes (all other B are zero), only the token ``far`` later reads (all other C are zero): what
    comes out there is the decayed product and nothing anywhere else, whole and with a cut before the reader."""
    H, G, N, V = 2, 1, 32, 16
    T = far + 1
    x, b, c = np.zeros((T, H, V)), np.zeros((T, G, N)), np.zeros((T, G, N))
    x[:] = 1.0
    b[0, 0], c[far, 0] = np.arange(N) % 5 + 1.0, np.arange(N) % 3 - 0.5
    rows = torch.tensor(np.concatenate([x.reshape(T, -1), b.reshape(T, -1), c.reshape(T, -1)], axis=1), dtype=dtype, device=DEV)
    steps, bias, a_log = torch.full((T, H), -3.0, device=DEV), torch.zeros(H, device=DEV), f32([-6.0, -1.5])
    want = ssd_want(rows, steps, bias, a_log, H, G, N, V)
    assert np.abs(want[far]).max() > 0.1
    for sizes in ([T], [T - 1, 1]):
        state = torch.zeros(1, H * N * V, device=DEV)
        at, got = 0, []
        for n in sizes:
            got.append(npy(run_ssd(rows, steps, bias, a_log, H, G, N, V, [n], [at], [0], state)[0]))
            at += n
        got = np.concatenate(got)
        assert np.abs(got[far] - want[far]).max() < 1e-4 and np.abs(got[:far]).max() == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,V,parts", [(6, 16, 2), (5, 14, 7), (4, 64, 4), (2, 24, 1), (32, 64, 64), (3, 20, 60)])
def test_state_space_output(dtype, H, V, parts):
    """The skip, then the gate, then the norm in parts of very different sizes, each by its own root mean square."""
    g = torch.Generator(device=DEV).manual_seed(7)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    n, inner = 7, H * V
    sizes = torch.tensor([10.0 ** (i % 3 - 1) for i in range(parts)], device=DEV).repeat_interleave(inner // parts)
    o, d, w = rnd(n, inner) * sizes, rnd(H), rnd(inner) + 1.0
    wide = (rnd(n, 2 * inner + 8) * torch.cat([sizes, torch.ones(8, device=DEV), torch.ones(inner, device=DEV)])).to(dtype)
    v, z = wide[:, :inner], wide[:, inner + 8:]
    out = torch.empty(n, inner, dtype=dtype, device=DEV)
    kernels.ssd_output(o, v, z, d, w, parts, 1e-5, out, V)
    y = (npy(o) + np.repeat(npy(d), V) * npy(v)) * plain.silu(npy(z))
    want = plain.rms_unit(y.reshape(n, parts, -1), 1e-5).reshape(n, inner) * npy(w)
    np.testing.assert_allclose(npy(out), want, **(dict(rtol=3e-5, atol=3e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)))


# ---- the recurrence's gates on tensor cores ----------------------------------------------------------------------------


@pytest.mark.parametrize("n,width,blocks", [(129, 64, 4), (200, 96, 2), (150, 128, 1), (333, 240, 3), (64, 512, 2)])
def test_gates_of_bfloat16_matrices_equal_the_float_products(n, width, blocks):
    """u of many sizes, whose low bits weigh in: large entries that cancel in the product, beside small ones."""
    g = torch.Generator(device=DEV).manual_seed(10)
    bw = width // blocks
    u = torch.randn(n, width, generator=g, device=DEV) * 10.0 ** torch.randint(-2, 2, (n, width), generator=g, device=DEV)
    ra, ri = ((torch.randn(blocks, bw, bw, generator=g, device=DEV) * 0.2).bfloat16() for _ in range(2))
    for m in (ra, ri):
        m[:, :, 1] = -m[:, :, 0]
    u[:, 1::bw] = u[:, 0::bw] * (1 + 2.0 ** -12)
    u[:, 0::bw] *= 1.0
    ra_b, ri_b, lam = (torch.randn(width, generator=g, device=DEV) for _ in range(3))
    a, bx, a0, bx0 = (torch.empty(n, width, device=DEV) for _ in range(4))
    kernels.rglru_gates(u, ra, ra_b.view(blocks, bw), ri, ri_b.view(blocks, bw), lam, 8.0, a, bx)
    kernels.rglru_gates(u, ra.float(), ra_b.view(blocks, bw), ri.float(), ri_b.view(blocks, bw), lam, 8.0, a0, bx0)
    parts = npy(u).reshape(n, blocks, bw)
    gate = lambda m, b: plain.sigmoid(np.einsum("tbi,boi->tbo", parts, npy(m)).reshape(n, width) + npy(b))
    log_a = -8.0 * gate(ra, ra_b) * plain.softplus(npy(lam))
    want_a, want_b = np.exp(log_a), np.sqrt(-np.expm1(2 * log_a)) * gate(ri, ri_b) * npy(u)
    for got_a, got_b in ((a, bx), (a0, bx0)):
        np.testing.assert_allclose(npy(got_a), want_a, rtol=2e-4, atol=2e-6)
        np.testing.assert_allclose(npy(got_b), want_b, rtol=2e-4, atol=2e-6)


# ---- the latents ----------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels", [7, 64, 88, 1536])
def test_query_latent_norm_and_output_gate(dtype, channels):
    g = torch.Generator(device=DEV).manual_seed(8)
    wide = (torch.randn(11, channels + 8, generator=g, device=DEV) * 3).to(dtype)
    w = torch.randn(channels, generator=g, device=DEV) + 1.0
    out = torch.empty(11, channels, dtype=dtype, device=DEV)
    down, dw = torch.randn(11, 20, generator=g, device=DEV).to(dtype), torch.ones(12, device=DEV)
    pages = torch.zeros(2, 1, 8, 20, dtype=dtype, device=DEV)
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    for own in (True, False):                                   # with and without a cache row of its own
        out.zero_()
        kernels.latent_store(down, 12, 8, dw, 1e-2, None, "interleaved", pages if own else None, i32(np.arange(11) + 3), wide[:, 3:3 + channels], w, out)
        np.testing.assert_allclose(npy(out), plain.rms_unit(npy(wide[:, 3:3 + channels]), 1e-2) * npy(w), **tol)
    row = np.concatenate([plain.rms_unit(npy(down)[:, :12], 1e-2), npy(down)[:, 12:]], axis=1)
    np.testing.assert_allclose(npy(pages).reshape(16, 20)[3:14], row, **tol)
    assert (pages.view(16, 20)[:3] == 0).all() and (pages.view(16, 20)[14:] == 0).all()
    y = torch.randn(11, channels, generator=g, device=DEV).to(dtype)
    for off in (5, 4):                                          # rows that start where four channels can be read at once, and not
        want = npy(y) * plain.sigmoid(npy(wide[:, off:off + channels]))
        kernels.sigmoid_gate(y, wide[:, off:off + channels])
        np.testing.assert_allclose(npy(y), want, **tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank,rot", [(5, 64, 32), (3, 24, 12), (20, 64, 32), (16, 128, 64)])
def test_one_far_latent_carries_the_weight(dtype, heads, rank, rot):
    """Queries of runs and of single tokens whose score on one cached row stands out by 30 among hundreds: the first row, rows
    at a page's border, the row of the token itself; a row beyond the token (a later one of its own run) made to stand
    out by more must stay unseen."""
    g = torch.Generator(device=DEV).manual_seed(9)
    page, D = 8, rank + rot
    entries = [(300, 1), (0, 70), (37, 5), (63, 1), (0, 1)]            # tokens in the cache, tokens of the step
    peaks = {0: {0: 0}, 1: {69: 0, 40: 16, 8: 7, 7: 8, 0: 1}, 2: {0: 31, 4: 32, 2: 39}, 3: {0: 63}}
    total = [s + n for s, n in entries]
    keys = [torch.randn(t, D, generator=g, device=DEV) * 0.3 for t in total]
    qs = [torch.randn(n, heads, D, generator=g, device=DEV) * 0.3 for _, n in entries]
    for e, at in peaks.items():
        for t, j in at.items():
            unit = torch.zeros(D, device=DEV)
            unit[(5 * j + 3 * e) % D] = 1.0
            keys[e][j] += 4.0 * unit
            qs[e][t] += 30.0 * unit
    n_pages = [-(-t // page) for t in total]
    order = np.random.default_rng(3).permutation(sum(n_pages))
    pages = torch.full((sum(n_pages), 1, page, D), 100.0, device=DEV)           # what no token wrote must never weigh in
    table, slots, used = np.zeros((len(entries), max(n_pages)), dtype=np.int64), [], 0
    for e, t in enumerate(total):
        own = order[used:used + n_pages[e]]
        used += n_pages[e]
        table[e, :len(own)] = own
        for j in range(t):
            pages[own[j // page], 0, j % page] = keys[e][j]
    pages = pages.to(dtype)
    q = torch.cat(qs).reshape(-1, heads * D).to(dtype)
    lens = [n for _, n in entries]
    host = HostStep(lens, [s for s, _ in entries], sum(lens), len(lens))
    plan = {k: (i32(v) if len(v) else None) for k, v in attention_ops.plan_biased(host, heads, 0, 0).items()}
    ctx = SimpleNamespace(cu_q=i32(np.cumsum([0] + lens)), q_start_pos=i32([s for s, _ in entries]), token_seq=i32(np.repeat(np.arange(len(lens)), lens)),
                          n_seqs=len(lens), max_kv_len=max(total))
    kv = KVStep(pages, pages, None, i32(table), page)
    got = npy(attention_ops.attend_biased(ctx, plan, q, kv, heads, 1, D, rank, None, 0, 0.25, None, None, None, v_row=D)).reshape(-1, heads, rank)
    at = 0
    for e, (s, n) in enumerate(entries):
        k = npy(keys[e].to(dtype))
        for t in range(n):
            seen = k[:s + t + 1]
            qq = npy(q[at + t].reshape(heads, D))
            sc = qq @ seen.T * 0.25
            p = np.exp(sc - sc.max(axis=1, keepdims=True))
            p /= p.sum(axis=1, keepdims=True)
            want = p @ seen[:, :rank]
            assert np.abs(got[at + t] - want).max() < (2e-4 if dtype == torch.float32 else 4e-2), f"entry {e} token {t}"
        at += n

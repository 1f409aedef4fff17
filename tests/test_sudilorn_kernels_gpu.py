"""The kernels of the Sudilorn design's mechanisms, each alone against plain float64 arithmetic, with inputs made so that a
fault shows: a key on one map of one head that stands out among hundreds, just inside and just outside the window; the two
maps far apart; keys of a memory that repeat, so that what was written before must be taken back; a memory that never
forgets and one that forgets at once; groups whose two largest numbers beat another's largest; corrections that must not
weigh; updates scaled by vectors with signs."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import sudilorn as plain
from qwen25vl_lite.engine.runner import HostStep, KVStep
from qwen25vl_lite.ops import attention as attention_ops
from qwen25vl_lite.ops import delta_rule, kernels
from qwen25vl_lite.ops.linear import DeferredNorm, Linear
from qwen25vl_lite.parts.feed_forward import GroupedRoutedMLP

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)
f32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)
npy = lambda t: t.detach().double().cpu().numpy()
close = lambda dtype, tight=2e-5, loose=1e-2: dict(rtol=tight, atol=tight) if dtype == torch.float32 else dict(rtol=loose, atol=loose)


def generator(seed):
    g = torch.Generator(device=DEV).manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, device=DEV)


# ---- updates scaled per channel on their way into the stream --------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [96, 100, 2048, 77])
def test_scaled_update_then_norm(dtype, width):
    """x += s * update, then the norm of the sum with its weight; on chosen rows, which leave the stream as it is; the
    addition alone."""
    rnd = generator(1)
    x, y, s, w = rnd(7, width) * 3, rnd(7, width).to(dtype), rnd(width), rnd(width) * 0.3 + 1.0
    new = npy(x) + npy(s) * npy(y)
    x1, out = x.clone(), torch.empty(7, width, dtype=dtype, device=DEV)
    kernels.add_norm_groups(x1, y, s, 0.0, 0, w, 1e-5, 1, out)
    np.testing.assert_allclose(npy(x1), new, rtol=1e-5, atol=1e-5)
    np.testing.assert_allclose(npy(out), plain.rms_unit(new, 1e-5) * npy(w), **close(dtype))
    x2, some = x.clone(), torch.empty(2, width, dtype=dtype, device=DEV)
    kernels.add_norm_groups(x2, y, s, 0.0, 0, w, 1e-5, 1, some, i32([4, 1]))
    assert torch.equal(x2, x)
    np.testing.assert_allclose(npy(some), (plain.rms_unit(new, 1e-5) * npy(w))[[4, 1]], **close(dtype))
    kernels.add_norm_groups(x2, y, s, 0.0, 0, None, 0.0, 1, None, dtype=dtype)
    np.testing.assert_allclose(npy(x2), new, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("rows,n,k", [(1, 96, 128), (8, 2048, 2048), (3, 100, 5632), (5, 4096, 11008), (8, 40, 32)])
def test_product_scaled_into_the_stream(rows, n, k):
    """A few rows through the weight-streaming kernel: the product times a vector is added into the float32 stream, with K in
    one piece and cut, with and without a norm in front; in a chain behind another product."""
    rnd = generator(2)
    x, w, s, stream = (rnd(rows, k) * 0.5).bfloat16(), (rnd(n, k) / k ** 0.5).bfloat16(), rnd(n), rnd(rows, n)
    got = stream.clone()
    assert Linear(w)(x, residual=got, residual_scale=s) is None
    want = npy(stream) + npy(s) * (npy(x) @ npy(w).T)
    np.testing.assert_allclose(npy(got), want, rtol=1e-4, atol=1e-4)
    norm_w, xf = rnd(k) * 0.2 + 1.0, rnd(rows, k)
    got = stream.clone()
    assert Linear(w)(DeferredNorm(xf, norm_w, 1e-5, torch.bfloat16), residual=got, residual_scale=s) is None
    want = npy(stream) + npy(s) * ((plain.rms_unit(npy(xf), 1e-5) * npy(norm_w)) @ npy(w).T)
    np.testing.assert_allclose(npy(got), want, rtol=2e-2, atol=2e-2)
    if n % 32 == 0:
        second = Linear((rnd(64, n) / n ** 0.5).bfloat16())
        chained, alone = stream.clone(), stream.clone()
        assert kernels.chain_begin()
        try:
            Linear(w)(x, residual=chained, residual_scale=s)
            y1 = second(DeferredNorm(chained, torch.ones(n, device=DEV), 1e-5, torch.bfloat16))
        finally:
            kernels.chain_end()
        Linear(w)(x, residual=alone, residual_scale=s)
        y2 = second(DeferredNorm(alone, torch.ones(n, device=DEV), 1e-5, torch.bfloat16))
        np.testing.assert_allclose(npy(chained), npy(alone), rtol=1e-5, atol=1e-5)
        np.testing.assert_allclose(npy(y1), npy(y2), rtol=2e-2, atol=2e-2)


# ---- queries and keys on their way into the cache ---------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dk,dv,dims,layout,scaled", [(6, 3, 20, 28, 12, "halves", True), (4, 1, 32, 64, 32, "halves", True), (2, 2, 64, 128, 20, "halves", False),
                                                               (5, 1, 128, 128, 128, "interleaved", False), (3, 3, 7, 10, 0, "halves", False),
                                                               (4, 2, 64, 64, 64, "interleaved", True), (8, 2, 48, 32, 16, "halves", False)])
def test_queries_normed_turned_and_two_maps_cached_side_by_side(dtype, heads, kv, dk, dv, dims, layout, scaled):
    """Every map of a head over its root mean square times a weight, its first channels turned by the token's position; the
    key rows of the cache hold both maps; values as they are; nothing else of the pages is touched."""
    rnd = generator(3)
    n, page, nq, nkv = 13, 8, 2 * heads, 2 * kv
    rot = {"dims": dims, "base": 300.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0} if scaled else None}
    width = (nq + nkv) * dk + kv * dv
    rows = (rnd(n, width + 6) * 2).to(dtype)[:, 2:2 + width] if dk % 2 else (rnd(n, width + 8) * 2).to(dtype)[:, :width]
    wq, wk = rnd(dk) * 0.3 + 1.0, rnd(dk) * 0.3 + 1.0
    first = 1000
    freqs, mag = plain.ramp_frequencies(dims, 300.0, rot["scaling"]) if dims else (np.zeros(0), 1.0)
    angles = kernels.rotary_angles(i32(np.arange(n) + first), f32(freqs), mag) if dims else None
    slots = torch.randperm(5 * page, generator=torch.Generator().manual_seed(3))[:n].to(torch.int32).to(DEV)
    kp, vp = torch.full((5, kv, page, 2 * dk), 9.0, dtype=dtype, device=DEV), torch.full((5, kv, page, dv), 9.0, dtype=dtype, device=DEV)
    raw = npy(rows)
    kernels.qk_norm_store(rows, wq, wk, 1e-5, angles, layout, kp, vp, slots, nq, nkv, dk, page, False, unit_norm=True, dv=dv, pack=2)

    def turned(x, weight):
        x = plain.rms_unit(x, 1e-5) * npy(weight)
        if not dims:
            return x
        padded = np.concatenate([np.zeros((first, *x.shape[1:])), x])
        return plain.rotate(padded, rot, "halves" if layout == "halves" else "pairs")[first:]

    tol = close(dtype, 2e-3, 3e-2)              # an angle of position 1,000 carries a thousand times its frequency's rounding
    np.testing.assert_allclose(npy(rows)[:, :nq * dk].reshape(n, nq, dk), turned(raw[:, :nq * dk].reshape(n, nq, dk), wq), **tol)
    page_of, at = (slots // page).long(), (slots % page).long()
    want_k = turned(raw[:, nq * dk:(nq + nkv) * dk].reshape(n, nkv, dk), wk).reshape(n, kv, 2 * dk)
    np.testing.assert_allclose(npy(kp[page_of, :, at]), want_k, **tol)
    np.testing.assert_array_equal(npy(vp[page_of, :, at]).reshape(n, -1), raw[:, (nq + nkv) * dk:])
    touched = torch.zeros(5, page, dtype=torch.bool, device=DEV)
    touched[page_of, at] = True
    assert (kp.transpose(1, 2)[~touched] == 9.0).all() and (vp.transpose(1, 2)[~touched] == 9.0).all()


# ---- differential attention --------------------------------------------------------------------------------------------


class PagedCase:
    """Keys and values of a few requests in shuffled pages (what no token wrote is large, so that it must never weigh in), the
    queries and gates of one step, and the step's context."""

    def __init__(self, dtype, entries, kv, key_width, dv, page, seed):
        self.rnd, self.entries, self.page, self.kv = generator(seed), entries, page, kv
        self.total = [s + n for s, n in entries]
        self.keys = [self.rnd(t, kv, key_width) * 0.3 for t in self.total]
        self.values = [self.rnd(t, kv, dv) for t in self.total]
        self.dtype, self.seed = dtype, seed

    def place(self):
        counts = [-(-t // self.page) for t in self.total]
        order = np.random.default_rng(self.seed).permutation(sum(counts))
        kp = torch.full((sum(counts), self.kv, self.page, self.keys[0].shape[2]), 100.0, device=DEV)
        vp = torch.full((sum(counts), self.kv, self.page, self.values[0].shape[2]), 100.0, device=DEV)
        table, used = np.zeros((len(counts), max(counts)), dtype=np.int64), 0
        for e, t in enumerate(self.total):
            own = order[used:used + counts[e]]
            used += counts[e]
            table[e, :len(own)] = own
            for j in range(t):
                kp[own[j // self.page], :, j % self.page] = self.keys[e][j]
                vp[own[j // self.page], :, j % self.page] = self.values[e][j]
        self.kv_step = KVStep(kp.to(self.dtype), vp.to(self.dtype), None, i32(table), self.page)
        lens, starts = [n for _, n in self.entries], [s for s, _ in self.entries]
        self.lens, self.host = lens, HostStep(lens, starts, sum(lens), len(lens))
        self.ctx = SimpleNamespace(cu_q=i32(np.cumsum([0] + lens)), q_start_pos=i32(starts), token_seq=i32(np.repeat(np.arange(len(lens)), lens)),
                                   n_seqs=len(lens), max_kv_len=max(self.total))

    def plan(self, group, window, keep, wide=False):
        """``wide``: with the row tiles of the tcgen05 kernels."""
        lists = attention_ops.plan_biased(self.host, group, window or 0, keep)
        if wide:
            lists["tiles128"] = attention_ops.plan_step(self.host, group, window or 0, 0)["tiles128"]
        return {k: (i32(v) if len(v) else None) for k, v in lists.items()}


def differential_case(dtype, heads, kv, dk, dv, page, window, entries, peaks, seed, lam=0.6, diff=0.4, scale=0.25, wide=None):
    """``peaks``: (entry, token of the step, head, map, key): that map's score on that key stands out by far.  Returns the
    kernels' result and the float64 one, [tokens, heads, dv]."""
    case = PagedCase(dtype, entries, kv, 2 * dk, dv, page, seed)
    group = heads // kv
    wide = (dk, dv) == (64, 128) and 128 % (2 * group) == 0 if wide is None else wide
    qs = [case.rnd(n, heads, 2, dk) * 0.3 for _, n in entries]
    for e, t, h, m, j in peaks:
        unit = torch.zeros(dk, device=DEV)
        unit[(5 * j + 3 * h + m) % dk] = 1.0
        case.keys[e][j, h // group, m * dk:(m + 1) * dk] += 4.0 * unit
        qs[e][t, h, m] += 30.0 * unit
    case.place()
    n = sum(case.lens)
    q = torch.cat(qs).to(dtype)
    # the kernels' order: by kv head, map, head of the group; the row goes on behind the queries
    rows = torch.cat([q.view(n, kv, group, 2, dk).transpose(2, 3).reshape(n, -1), torch.zeros(n, 8 if wide else 10, dtype=dtype, device=DEV)], dim=1)
    pad = 8 if wide else 6
    gate = torch.cat([torch.zeros(n, pad, dtype=dtype, device=DEV), case.rnd(n, heads * dv).to(dtype)], dim=1)[:, pad:]
    if dtype == torch.bfloat16 and wide:
        assert kernels.differential_attention_tcgen05_supports(rows, gate, heads, kv, dk, dv, page)
    got = attention_ops.attend_differential(case.ctx, case.plan(2 * group, window, 0, wide), rows, gate, case.kv_step, heads, kv, dk, dv, window, scale, lam, 1.0 - diff, 1e-5)
    at, want = 0, []
    for e, (s, m) in enumerate(entries):
        k, v = npy(case.keys[e].to(dtype)).reshape(s + m, kv, 2, dk), npy(case.values[e].to(dtype))
        seen = plain.visible(s + m, {"size": window} if window else None)[s:]
        qq = npy(q[at:at + m])
        heads_of = lambda a: np.stack([plain.softmax_attention(qq[:, h, a], k[:, h // group, a], v[:, h // group], scale, seen) for h in range(heads)], axis=1)
        want.append(plain.differential_heads(heads_of(0), heads_of(1), lam, diff, 1e-5))
        at += m
    return npy(got).reshape(n, heads, dv), np.concatenate(want) * plain.sigmoid(npy(gate)).reshape(n, heads, dv)


DIFF_SIZES = [(4, 2, 32, 64, 16), (6, 3, 20, 28, 8), (8, 1, 64, 128, 16), (4, 4, 64, 128, 8), (4, 2, 64, 128, 4), (16, 1, 64, 128, 16), (5, 1, 64, 128, 16), (5, 1, 128, 128, 32), (10, 1, 32, 32, 16), (20, 2, 64, 64, 16), (2, 2, 128, 32, 8), (3, 1, 7, 10, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dk,dv,page", DIFF_SIZES)
def test_differential_attention_at_the_windows_edges(dtype, heads, kv, dk, dv, page):
    """Keys that would carry a map's whole weight, at the last place a query sees and at the first that it does not, on the
    first map, the second, and both; in runs and for single tokens; at page borders; a token's own key and the next one's."""
    window = 37
    entries = [(150, 1), (0, 70), (61, 1), (30, 45), (0, 1), (36, 1), (100, 2), (70, 300)]
    peaks = [(7, 299, 0, 0, 369 - 36), (7, 298, 1, 1, 368 - 37), (7, 127, 0, 1, 197 - 36), (7, 128, 1, 0, 198), (0, 0, 0, 0, 150 - 36), (0, 0, 1, 1, 150 - 37), (1, 69, 0, 0, 33), (1, 68, 1, 1, 31), (1, 40, 0, 1, 16), (1, 41, 1, 0, 16), (1, 36, 0, 0, 0), (1, 37, 1, 1, 0),
             (2, 0, 0, 1, 61 - 36), (2, 0, 1, 0, 61 - 37), (3, 10, 0, 0, 4), (3, 11, 1, 1, 4), (3, 44, 0, 1, 74), (3, 20, 1, 0, 51), (5, 0, 0, 0, 0), (6, 1, 0, 1, 65), (6, 0, 1, 0, 63)]
    peaks = [p for p in peaks if p[2] < heads]
    got, want = differential_case(dtype, heads, kv, dk, dv, page, window, entries, peaks, 4)
    # the difference of the maps is divided by its own size: bfloat16's rounding of the weights shows where it is small
    assert np.abs(got - want).max() < (2e-4 if dtype == torch.float32 else 6e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dk,dv,page", [(4, 2, 32, 64, 16), (4, 1, 64, 128, 16), (2, 1, 20, 24, 8)])
def test_differential_attention_over_everything(dtype, heads, kv, dk, dv, page):
    """No window: a far key on one map among a thousand, in single tokens whose keys are cut into ranges, and in runs."""
    entries = [(1100, 1), (700, 40), (0, 130)]
    peaks = [(0, 0, 0, 0, 3), (0, 0, 1, 1, 1100), (1, 39, 0, 1, 15), (1, 0, 1, 0, 16), (2, 129, 0, 0, 0), (2, 63, 1, 1, 64 - 1)]
    got, want = differential_case(dtype, heads, kv, dk, dv, page, None, entries, peaks, 5, lam=1.3, diff=0.15)
    assert np.abs(got - want).max() < (2e-4 if dtype == torch.float32 else 6e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dk,dv", [(32, 64), (64, 128)])
def test_differential_attention_is_each_request_alone(dtype, dk, dv):
    """Bit for bit: a request's rows do not depend on the others of its step."""
    heads, kv, page, window = 4, 2, 16, 50
    wide = (dk, dv) == (64, 128)
    entries = [(150, 1), (0, 70), (61, 1), (30, 45)]
    together, _ = differential_case(dtype, heads, kv, dk, dv, page, window, entries, [], 6)
    lone = PagedCase(dtype, entries, kv, 2 * dk, dv, page, 6)
    qs = [lone.rnd(n, heads, 2, dk) * 0.3 for _, n in entries]
    lone.place()
    n = sum(lone.lens)
    rows = torch.cat(qs).to(dtype).view(n, kv, heads // kv, 2, dk).transpose(2, 3).reshape(n, -1).contiguous()
    gate = lone.rnd(n, heads * dv).to(dtype)
    at = 0
    for e, (s, m) in enumerate(entries):
        host = HostStep([m], [s], m, 1)
        ctx = SimpleNamespace(cu_q=i32([0, m]), q_start_pos=i32([s]), token_seq=i32([0] * m), n_seqs=1, max_kv_len=lone.ctx.max_kv_len)
        lists = attention_ops.plan_biased(host, 2 * heads // kv, window, 0)
        if wide:
            lists["tiles128"] = attention_ops.plan_step(host, 2 * heads // kv, window, 0)["tiles128"]
        plan = {k: (i32(v) if len(v) else None) for k, v in lists.items()}
        kv_step = KVStep(lone.kv_step.k_pages, lone.kv_step.v_pages, None, lone.kv_step.block_table[e:e + 1].contiguous(), page)
        got = attention_ops.attend_differential(ctx, plan, rows[at:at + m], gate[at:at + m], kv_step, heads, kv, dk, dv, window, 0.25, 0.6, 0.6, 1e-5)
        np.testing.assert_array_equal(npy(got).reshape(m, heads, dv), together[at:at + m])
        at += m


# ---- window attention with kept first tokens into strided rows ----------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,dk,dv,page,window,keep", [(4, 2, 64, 64, 16, 20, 5), (6, 2, 24, 20, 8, 9, 3), (8, 8, 128, 128, 16, 64, 20), (4, 1, 32, 128, 8, 4, 9),
                                                           (2, 1, 128, 128, 32, 33, 40), (20, 1, 64, 32, 16, 12, 2), (4, 1, 128, 128, 16, 70, 66), (16, 2, 128, 128, 16, 150, 4),
                                                           (3, 1, 128, 128, 4, 90, 130), (4, 2, 128, 128, 16, 64, 0)])
def test_window_and_kept_tokens_into_columns_of_wider_rows(dtype, nq, nkv, dk, dv, page, window, keep):
    """Keys that carry the whole weight as the last kept token, the first that is not kept, the last the window shows and the
    first it does not; the result goes into columns of wider rows and leaves the others alone."""
    entries = [(100, 1), (0, 90), (40, 1), (50, 30), (0, 1), (120, 260)]
    group, tiles128 = nq // nkv, dk == 128 and dv == 128          # those runs go to the tcgen05 kernel
    assert not tiles128 or attention_ops.tcgen05_runs(dk, dv, group, window, keep, None, 0, 0.0)
    case = PagedCase(dtype, entries, nkv, dk, dv, page, 7)
    qs = [case.rnd(n, nq, dk) * 0.3 for _, n in entries]
    places = lambda p: (keep - 1, keep, p - window + 1, p - window, p, 0)
    for e, t in ((0, 0), (1, 89), (1, 60), (2, 0), (3, 3), (3, 29), (5, 259), (5, 100), (5, 64)):
        p = entries[e][0] + t
        for h, j in enumerate(places(p)[:nq]):
            if 0 <= j <= p:
                unit = torch.zeros(dk, device=DEV)
                unit[(5 * j + 3 * h) % dk] = 1.0
                case.keys[e][j, h // group] += 4.0 * unit
                qs[e][t, h] += 30.0 * unit
    case.place()
    n = sum(case.lens)
    q = torch.cat(qs).to(dtype)
    wide = torch.full((n, nq * dv + 24), 7.0, dtype=dtype, device=DEV)
    attention_ops.attend_biased(case.ctx, case.plan(group, window, keep, tiles128), q.reshape(n, -1), case.kv_step, nq, nkv, dk, dv, window, keep, 0.25, None, None, out=wide[:, 16:16 + nq * dv])
    assert (wide[:, :16] == 7.0).all() and (wide[:, 16 + nq * dv:] == 7.0).all()
    got, at = npy(wide[:, 16:16 + nq * dv]).reshape(n, nq, dv), 0
    for e, (s, m) in enumerate(entries):
        k, v = npy(case.keys[e].to(dtype)), npy(case.values[e].to(dtype))
        seen = plain.visible(s + m, {"size": window, "keep_first": keep})[s:]
        qq = npy(q[at:at + m])
        want = np.stack([plain.softmax_attention(qq[:, h], k[:, h // group], v[:, h // group], 0.25, seen) for h in range(nq)], axis=1)
        assert np.abs(got[at:at + m] - want).max() < (2e-4 if dtype == torch.float32 else 4e-2), f"entry {e}"
        at += m


# ---- the gated delta rule ----------------------------------------------------------------------------------------------


def portions_of(total, sizes):
    out, k = [], 0
    while sum(out) < total:
        out.append(min(sizes[k % len(sizes)], total - sum(out)))
        k += 1
    return out


def delta_case(dtype, H, G, D, V, total, seed):
    """Rows q | k | v, gates and per-head constants: head 0 keeps everything, head 1 forgets at once, the others are in
    between; every third key is close to an earlier one; write strengths cover (0, 1)."""
    rnd = generator(seed)
    rows = rnd(total, 2 * G * D + H * V)
    k = rows[:, G * D:2 * G * D]
    for t in range(6, total, 3):
        k[t] = k[t - 5] * 1.5 + 0.1 * rnd(G * D)
    gates = rnd(total, 2 * H) * 1.5
    bias = rnd(H) * 0.3 - 2.0
    a_log = torch.linspace(-3.0, 1.0, H, device=DEV)
    a_log[0] = -15.0
    if H > 1:
        a_log[1] = 3.0
    return rows.to(dtype), gates, bias, a_log


def delta_want(rows, gates, bias, a_log, H, G, D, V):
    T, r = rows.shape[0], npy(rows)
    of_head = np.arange(H) // (H // G)
    q, k = (plain.unit_vectors(x.reshape(T, G, D))[:, of_head] for x in (r[:, :G * D], r[:, G * D:2 * G * D]))
    z = npy(gates)
    decay = np.exp(-np.exp(npy(a_log)) * plain.softplus(z[:, :H] + npy(bias)))
    return plain.delta_rule(q * D ** -0.5, k, r[:, 2 * G * D:].reshape(T, H, V), plain.sigmoid(z[:, H:]), decay)


def run_delta(case, H, G, D, V, lens, starts, slots, state, tensor_cores=True):
    """One step over entries (their first rows in ``starts``): float32 results per entry, without the output's norm and gate."""
    rows, gates, bias, a_log = case
    x = torch.cat([rows[s:s + n] for s, n in zip(starts, lens)]).contiguous()
    z = torch.cat([gates[s:s + n] for s, n in zip(starts, lens)]).contiguous()
    o = torch.empty(x.shape[0], H * V, device=DEV)
    mma = tensor_cores and kernels.delta_mma_supports(x.dtype, H, G, D, V)
    work = {k: (i32(v) if len(v) else None) for k, v in delta_rule.plan(list(lens), mma).items()}
    if work["runs"] is not None:
        kernels.delta_runs_mma(x, z, bias, a_log, state, i32(slots), o, work["chunks"], work["runs"], H, G, D, V, D ** -0.5, 1e-6)
    if work["runs"] is None or work["walked"] is not None:
        kernels.delta_walk(x, z, bias, a_log, state, i32(np.cumsum([0] + list(lens))), i32(slots), len(lens), work["walked"], o, H, G, D, V, D ** -0.5, 1e-6)
    return [t.view(-1, H, V) for t in torch.split(o, list(lens))]


DELTA_SIZES = [(4, 2, 32, 16), (6, 3, 24, 20), (5, 5, 10, 14), (3, 1, 128, 64), (2, 1, 64, 64), (4, 4, 128, 128), (2, 1, 96, 136), (8, 2, 64, 32), (6, 6, 32, 56), (6, 2, 128, 40),
               (1, 1, 13, 7), (2, 1, 256, 64), (1, 1, 300, 33), (2, 2, 64, 200), (40, 20, 64, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", DELTA_SIZES)
def test_delta_rule_whole_cut_and_decoded(dtype, H, G, D, V):
    """The same request whole, in portions from one token to several chunks, and token by token at its end: chunks on tensor
    cores, the walk and single tokens give the plain result, and leave the same state; what lies behind it stays."""
    total = 210
    case = delta_case(dtype, H, G, D, V, total, 8)
    want, end = delta_want(*case, H, G, D, V)
    scale = np.abs(want).max(axis=(0, 2))[:, None]
    tol = 3e-5 if dtype == torch.float32 else 3e-4
    behind = 8 + -(H * D * V) % 4
    for sizes, cores in (([total], True), ([total], False), ([50, 1, 1, 2, 64, 65, 27], True), ([130] + [1] * 80, True), ([15, 16, 17, 127, 35], True)):
        sizes = portions_of(total, sizes)
        state = torch.zeros(2, H * D * V + behind, device=DEV)
        state[:, H * D * V:] = 5.0
        at, got = 0, []
        for n in sizes:
            got.append(npy(run_delta(case, H, G, D, V, [n], [at], [1], state, cores)[0]))
            at += n
        # the inputs are the rounded ones on both sides; behind them everything is float32 or carries 16 bits
        assert (np.abs(np.concatenate(got) - want) / scale).max() < tol, f"portions {sizes}, tensor cores {cores}"
        assert (state[0, :H * D * V] == 0).all() and (state[:, H * D * V:] == 5.0).all()
        np.testing.assert_allclose(npy(state[1, :H * D * V]).reshape(H, D, V), end, rtol=tol, atol=tol * np.abs(end).max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 32, 16), (3, 1, 128, 64), (16, 8, 64, 64), (2, 1, 20, 24)])
def test_delta_rule_batches_of_unequal_entries(dtype, H, G, D, V):
    """Long runs, short runs and single tokens of different requests in one step equal each alone, bit for bit."""
    case = delta_case(dtype, H, G, D, V, 700, 9)
    lens, starts, slots = [1, 300, 40, 129, 2, 128, 16], [0, 1, 301, 341, 470, 472, 600], [5, 0, 3, 1, 4, 2, 6]
    state = torch.randn(7, H * D * V + 4, generator=torch.Generator(device=DEV).manual_seed(1), device=DEV)
    before = state.clone()
    together = run_delta(case, H, G, D, V, lens, starts, slots, state)
    for i, (n, s, slot) in enumerate(zip(lens, starts, slots)):
        own = before.clone()
        alone = run_delta(case, H, G, D, V, [n], [s], [slot], own)[0]
        assert torch.equal(alone, together[i]) and torch.equal(own[slot], state[slot])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("far", [1, 15, 63, 64, 127, 128, 200])
def test_a_far_write_is_read_and_taken_back(dtype, far):
    """A first token writes along one key; the token ``far`` later reads it, the one after that writes another value along the
    same key with full strength, and the next reads only the new one.  The tokens between write along orthogonal keys."""
    H, G, D, V = 2, 1, 32, 16
    T = far + 3
    q, k, v = np.zeros((T, D)), np.zeros((T, D)), np.ones((T, H * V))
    k[:, 1] = 1.0
    k[0], k[far + 1] = 0.0, 0.0
    k[0, 0] = k[far + 1, 0] = 1.0
    q[far, 0] = q[far + 2, 0] = 2.0
    v[0], v[far + 1] = 3.0, -5.0
    rows = torch.tensor(np.concatenate([q, k, v], axis=1), dtype=dtype, device=DEV)
    gates = torch.cat([torch.full((T, H), -4.0), torch.full((T, H), 20.0)], dim=1).to(DEV)
    case = (rows, gates, torch.zeros(H, device=DEV), f32([-7.0, -1.0]))
    want, _ = delta_want(*case, H, G, D, V)
    assert abs(want[far, 0, 0]) > 0.4 and abs(want[far + 2, 0, 0] + 5.0 * D ** -0.5) < 0.01
    for sizes in ([T], [far, 3], [T - 1, 1]):
        state = torch.zeros(1, H * D * V, device=DEV)
        at, got = 0, []
        for n in sizes:
            got.append(npy(run_delta(case, H, G, D, V, [n], [at], [0], state)[0]))
            at += n
        assert np.abs(np.concatenate(got) - want).max() < 2e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 32, 16), (3, 1, 64, 128), (2, 2, 128, 128), (5, 5, 10, 14), (2, 1, 64, 200), (2, 1, 96, 136)])
def test_heads_are_finished_by_the_walk_and_behind_the_runs(dtype, H, G, D, V):
    """o / rms(o) * weight * silu(gate) per head into columns of wider rows: in the walk's own kernel where a head is one CTA's,
    and by the kernel behind the runs; results of very different sizes, so that a norm over the wrong channels shows."""
    case = delta_case(dtype, H, G, D, V, 90, 10)
    rows, gates, bias, a_log = case
    rows[:, 2 * G * D:] *= torch.tensor([10.0 ** (h % 3 - 1) for h in range(H)], device=DEV).repeat_interleave(V).to(dtype)
    want, _ = delta_want(rows, gates, bias, a_log, H, G, D, V)
    rnd = generator(11)
    w, wide_gate = rnd(V).repeat(H) + 1.0, rnd(90, H * V + 8).to(dtype)
    gate = wide_gate[:, 8:]
    full = plain.rms_unit(want, 1e-5).reshape(90, H * V) * npy(w) * plain.silu(npy(gate))
    for lens in ([1] * 90, [90], [7, 1, 60, 22]):
        state = torch.zeros(1, H * D * V + (-(H * D * V)) % 4, device=DEV)
        mma = kernels.delta_mma_supports(dtype, H, G, D, V)
        at = 0
        for n in lens:
            work = {k: (i32(a) if len(a) else None) for k, a in delta_rule.plan([n], mma).items()}
            ctx = SimpleNamespace(cu_q=i32([0, n]), slot_ids=i32([0]), n_seqs=1)
            wide = torch.full((n, H * V + 16), 7.0, dtype=dtype, device=DEV)
            delta_rule.run(work, ctx, rows[at:at + n].contiguous(), gates[at:at + n].contiguous(), bias, a_log, state, gate[at:at + n], w, 1e-5, wide[:, 8:8 + H * V],
                           H, G, D, V, D ** -0.5, 1e-6)
            assert (wide[:, :8] == 7.0).all() and (wide[:, 8 + H * V:] == 7.0).all()
            err = np.abs(npy(wide[:, 8:8 + H * V]) - full[at:at + n]) / (1.0 + np.abs(full[at:at + n]))
            assert err.max() < (2e-3 if dtype == torch.float32 else 1.5e-2), f"tokens {at} to {at + n}"
            at += n


# ---- routed experts without gates ---------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,count,keep,top", [(16, 2, 1, 4), (10, 5, 2, 3), (8, 1, 1, 2), (4, 4, 4, 4), (32, 8, 3, 6), (200, 100, 7, 5), (5, 5, 2, 1), (256, 4, 2, 16)])
def test_router_by_the_two_largest_of_a_group(dtype, experts, count, keep, top):
    """Choices and weights of 700 tokens (and of three) equal the plain router's; corrections of both signs, larger than the
    scores, never show in the weights; choosing by a group's largest number alone would choose otherwise."""
    rnd = generator(12)
    n, width = 700, 64
    h, router = rnd(n, width).to(dtype), rnd(experts, width) * 0.2
    corr = rnd(experts) * 0.5 - 0.5
    r = {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}
    z = npy(h) @ npy(router).T
    for rows in (n, 3):
        idx, w, counts = torch.empty(rows, top, dtype=torch.int32, device=DEV), torch.empty(rows, top, device=DEV), torch.zeros(experts, dtype=torch.int32, device=DEV)
        kernels.moe_route_softmax(h[:rows], router, corr, experts, top, count, keep, idx, w, counts, scores="sigmoid", mark="two_largest")
        same = 0
        for t in range(rows):
            chosen, weights = plain.route(z[t], npy(corr), r)
            if chosen.tolist() == idx[t].tolist():
                same += 1
                np.testing.assert_allclose(npy(w[t]), weights, rtol=1e-4, atol=1e-6)
        assert same >= 0.98 * rows                       # the rest: numbers within float32's rounding of one another
        assert counts.sum().item() == rows * top and torch.equal(torch.bincount(idx.reshape(-1).long(), minlength=experts).int(), counts)
        # the choice from logits that are there already, with and without counts
        idx2, w2, counts2 = torch.empty_like(idx), torch.empty_like(w), torch.zeros_like(counts)
        for c in (counts2, None):
            kernels.moe_choose(f32(z[:rows]), corr, experts, top, count, keep, idx2, w2, c, scores="sigmoid", mark="two_largest")
            agree = (idx2 == idx).all(dim=1)
            assert agree.float().mean() >= 0.98 and torch.allclose(w2[agree], w[agree], rtol=1e-4, atol=1e-6)
        assert torch.equal(torch.bincount(idx2.reshape(-1).long(), minlength=experts).int(), counts2)
    if 1 < count < experts and keep < count:
        other = torch.empty_like(idx)
        kernels.moe_route_softmax(h[:3], router, corr, experts, top, count, keep, other, w, counts, scores="sigmoid")
        marks = lambda k: [[np.sort(part)[::-1][:k].sum() for part in (plain.sigmoid(z[t]) + npy(corr)).reshape(count, -1)] for t in range(n)]
        assert any(np.argsort(a)[::-1][:keep].tolist() != np.argsort(b)[::-1][:keep].tolist() for a, b in zip(marks(1), marks(2)))


@pytest.mark.parametrize("pairs,experts,tile", [(1, 1, 16), (16, 8, 16), (2048, 256, 16), (2000, 7, 64), (300, 200, 128), (40, 33, 64)])
def test_pairs_sorted_by_one_block(pairs, experts, tile):
    """Every pair has a row of its own in its expert's tiles, the other rows are empty, and the tiles are its experts' in order;
    choices beyond the experts take no row; nothing has to be cleared before."""
    idx = torch.tensor(np.random.default_rng(3).integers(0, experts + 2, size=pairs) % (experts + 1), dtype=torch.int32, device=DEV)
    rows = kernels.moe_max_rows(pairs, experts, tile)
    plan, row_pair, pair_row = (torch.full((k,), 12345, dtype=torch.int32, device=DEV) for k in (2 + experts + rows // tile, rows, pairs))
    kernels.moe_sort_small(idx, plan, row_pair, pair_row, experts, tile)
    chosen, plan, row_pair, pair_row = (t.cpu().numpy() for t in (idx, plan, row_pair, pair_row))
    counts = np.bincount(chosen[chosen < experts], minlength=experts)
    tiles = -(-counts // tile)
    assert plan[0] == tiles.sum() and plan[1:2 + experts].tolist() == np.concatenate([[0], np.cumsum(tiles)]).__mul__(tile).tolist()
    assert plan[2 + experts:2 + experts + plan[0]].tolist() == np.repeat(np.arange(experts), tiles).tolist()
    for i in range(pairs):
        if chosen[i] == experts:
            assert pair_row[i] == -1
        else:
            assert row_pair[pair_row[i]] == i and plan[2 + experts + pair_row[i] // tile] == chosen[i]
    assert (row_pair >= 0).sum() == counts.sum() and (row_pair == -1).sum() == rows - counts.sum()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,experts,count,keep,top,width,ff", [(1, 8, 2, 1, 2, 64, 48), (7, 10, 5, 2, 3, 96, 40), (40, 4, 1, 1, 2, 100, 30), (300, 8, 4, 2, 2, 128, 72), (600, 4, 2, 1, 2, 256, 96),
                                                               (1100, 4, 2, 2, 2, 2048, 64)])
def test_routed_experts_with_and_without_the_stream(dtype, n, experts, count, keep, top, width, ff):
    """The weighted sum of squared-relu experts: as a result of its own, and scaled into the stream; steps of one token to
    steps whose experts get hundreds of rows (in bfloat16 the three kinds of grouped product)."""
    rnd = generator(13)
    part = GroupedRoutedMLP(width, experts, top, ff, count, keep)
    tensors = {}
    for ts in part.tensor_specs():
        tensors[ts.name] = (rnd(*ts.shape) * (0.05 if ts.name == "router" else ts.shape[-1] ** -0.5 * 1.5)).cpu()
    tensors["correction"] = torch.tensor(np.random.default_rng(1).permutation(np.linspace(-1.0, 1.0, experts)), dtype=torch.float32)
    tensors = {k: t.to(dtype).float() for k, t in tensors.items()}
    part.load(tensors, DEV, dtype)
    ctx = SimpleNamespace(dtype=dtype)
    h = rnd(n, width).to(dtype)
    want = plain.routed_ffn(npy(h), {k: npy(t) for k, t in tensors.items()}, {"router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}})
    size = np.abs(want).max()
    assert np.abs(npy(part.forward(ctx, h)) - want).max() < (2e-5 if dtype == torch.float32 else 1.5e-2) * size
    stream, scale = rnd(n, width), rnd(width)
    got = stream.clone()
    assert part.forward(ctx, h, residual=got, residual_scale=scale) is None
    assert np.abs(npy(got) - (npy(stream) + npy(scale) * want)).max() < (2e-5 if dtype == torch.float32 else 1.5e-2) * size * np.abs(npy(scale)).max()

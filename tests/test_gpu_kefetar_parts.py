"""Each Kefetar mechanism alone on the GPU against its plain function (tests/plain/kefetar_plain.py), on inputs made so that a
fault shows: the norm with one gain followed by a convolution and the convolution of a projection's columns, both over
schedules of prompts, portions and single tokens with one loud row whose echo ends exactly `taps` rows later, in slots that
held rubbish and slots used again; values blended between layers whose heads lie differently; retention with states that
barely decay, asked hundreds of tokens and several steps later for what was written at token 3; capped scores without a
sink in the attention kernels; the polynomial over normed powers, each power alone."""
import math

import numpy as np
import pytest
import torch

from tinyllama_c_b200 import ops
from tinyllama_c_b200.engine.step import chunk_table
from tinyllama_c_b200.parts.base import LayerCache, PartSpec
from plain import ops_plain
from plain import kefetar_plain as plain
from test_gpu_kernels import TOL as KTOL, _paged_setup, _step_arrays, cmp, gen, rnd

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dev(a, dtype=torch.float32):
    return torch.tensor(np.ascontiguousarray(a), dtype=dtype, device="cuda")


class _Step:
    """The packed batch of one step: counts of new rows, positions they start at, slots."""

    def __init__(self, counts, starts, slots, chunk_rows=None, chunk_from=None):
        self.n_seqs, self.n_rows, self.max_new = len(counts), sum(counts), max(counts)
        self.host_start = tuple(starts)
        self.cu_seqlens = dev(np.concatenate([[0], np.cumsum(counts)]), torch.int32)
        self.row_seq = dev(np.repeat(np.arange(len(counts)), counts), torch.int32)
        self.positions = dev(np.concatenate([s + np.arange(n) for s, n in zip(starts, counts)]), torch.int32)
        self.slots, self.start_pos = dev(slots, torch.int32), dev(starts, torch.int32)
        self.chunks, self.scratch = {}, {}
        if chunk_rows:
            tab = chunk_table(counts, chunk_rows, chunk_from)
            self.chunks[chunk_rows] = None if tab is None else tuple(dev(t, torch.int32) for t in tab)


def run_schedule(seqs, slots, cuts, call, **step_args):
    """seqs: arrays [T, C] (or tuples of them); cuts: the sizes of every sequence's portions.  call(rows, step) -> array of
    results for the packed rows; returns the results per sequence."""
    outs, at = [[] for _ in seqs], [0] * len(seqs)
    for s in range(max(len(c) for c in cuts)):
        live = [i for i in range(len(seqs)) if s < len(cuts[i])]
        counts = [cuts[i][s] for i in live]
        step = _Step(counts, [at[i] for i in live], [slots[i] for i in live], **step_args)
        rows = np.concatenate([seqs[i][at[i]:at[i] + n] for i, n in zip(live, counts)])
        y, o = call(rows, step), 0
        for i, n in zip(live, counts):
            outs[i].append(y[o:o + n])
            at[i] += n
            o += n
    return [np.concatenate(x) for x in outs]


# sizes of portions: whole prompts; portions shorter than a window, single tokens between them; single tokens from the start
SCHEDULES = [([70, 9, 1], [[70], [9], [1]]), ([41, 30], [[17, 1, 2, 1, 20], [1, 1, 3, 16, 9]]), ([12, 12, 12], [[1] * 12] * 3),
             ([40, 7], [[2] * 20, [1, 2, 2, 2]])]


# ---- convolutions ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("D,taps", [(5, 2), (52, 3), (64, 1), (100, 5), (1000, 4), (2048, 4), (4100, 17), (5000, 3)])
def test_norm_with_one_gain_and_its_convolution(dtype, D, taps):
    g = np.random.default_rng(taps)
    w = g.standard_normal((D, taps))
    w[:, 0] *= 3.0                              # the oldest tap speaks loudest: an echo one row short or long shows
    gain, eps = 1.37, 1e-5
    tol = 3e-5 if dtype == "float32" else 8e-3
    state = torch.full((5, max(taps - 1, 1), D), 7.0, device="cuda")        # slots that held rubbish
    wt, gv = dev(w.T), dev(np.full(D, gain))

    def call(rows, step):
        out = torch.empty(rows.shape, dtype=DT[dtype], device="cuda")
        ops.rmsnorm_conv(dev(rows), gv, eps, wt, state if taps > 1 else None, step, out)
        torch.cuda.synchronize()
        return out.float().cpu().numpy().astype(np.float64)

    for case, (lens, cuts) in enumerate(SCHEDULES):
        seqs = [(g.standard_normal((n, D)) * 0.05).astype(np.float32).astype(np.float64) for n in lens]
        for s in seqs:                          # rows so small that eps matters, one loud among them
            s[min(3, len(s) - 1)] *= 400.0
        slots = [3, 0, 2][:len(lens)] if case % 2 else [0, 3, 4][:len(lens)]
        got = run_schedule(seqs, slots, cuts, call)
        for i, s in enumerate(seqs):
            want = plain.sublayer_input(s, np.array(gain), w, eps)
            err = np.abs(got[i] - want).max(1)
            assert err.max() <= tol * np.abs(want).max(), f"case {case} sequence {i} row {int(err.argmax())}: {err.max():.3e}"


@pytest.mark.parametrize("C,off,pad,taps", [(48, 4, 8, 3), (45, 3, 2, 2), (512, 0, 0, 4), (36, 4, 4, 1), (64, 8, 4, 6), (1028, 0, 4, 3)])
def test_convolution_of_projected_columns(C, off, pad, taps):
    g = np.random.default_rng(C)
    w = g.standard_normal((C, taps))
    w[:, 0] *= 3.0
    state = torch.full((5, max(taps - 1, 1), C), 7.0, device="cuda")
    wt = dev(w.T)

    def call(rows, step):
        out = torch.empty((len(rows), C), device="cuda")
        ops.channel_conv(dev(rows), off, wt, state if taps > 1 else None, step, out)
        torch.cuda.synchronize()
        return out.cpu().numpy().astype(np.float64)

    for case, (lens, cuts) in enumerate(SCHEDULES):
        seqs = [g.standard_normal((n, off + C + pad)).astype(np.float32).astype(np.float64) for n in lens]
        for s in seqs:
            s[min(3, len(s) - 1)] *= 50.0
        got = run_schedule(seqs, ([3, 0, 2] if case % 2 else [0, 3, 4])[:len(lens)], cuts, call)
        for i, s in enumerate(seqs):
            want = plain.causal_conv(s[:, off:off + C], w)
            err = np.abs(got[i] - want).max(1)
            assert err.max() <= 1e-5 * np.abs(want).max(), f"case {case} sequence {i} row {int(err.argmax())}: {err.max():.3e}"


@pytest.mark.parametrize("heads,first_heads,n,n_first", [((24, 16), (24, 16), 2, 2), ((24, 16), (32, 32), 2, 1), ((32, 32), (8, 8), 1, 4),
                                                          ((64, 48), (64, 48), 2, 2), ((20, 20), (30, 10), 3, 6)])
def test_values_blended_between_layers(heads, first_heads, n, n_first):
    """Value by value, whatever columns the two layers' heads take; what lies past a head's values stays as it is."""
    g = np.random.default_rng(4)
    (hd, vd), (hd_f, vd_f) = heads, first_heads
    assert n * vd == n_first * vd_f
    T, q, lam = 19, 12, 0.3
    x = g.standard_normal((T, q + n * hd)).astype(np.float32)
    f = g.standard_normal((T, 8 + n_first * hd_f)).astype(np.float32)
    if heads == first_heads:
        x[:, q:].reshape(T, n, hd)[:, :, vd:] = 0.0
        f[:, 8:].reshape(T, n_first, hd_f)[:, :, vd_f:] = 0.0
    out = torch.empty((T, q + n * hd), device="cuda")
    fd = dev(f)
    ops.channel_conv(dev(x), 0, dev(np.full((1, q + n * hd), 2.0)), None, _Step([T], [0], [0]), out, fd[:, 8:], q, lam, heads, first_heads)
    got = out.cpu().numpy()
    want = 2.0 * x.astype(np.float64)
    own = want[:, q:].reshape(T, n, hd)
    flat = plain.mix_values(own[:, :, :vd].reshape(T, -1), f[:, 8:].astype(np.float64).reshape(T, n_first, hd_f)[:, :, :vd_f].reshape(T, -1), lam)
    own[:, :, :vd] = flat.reshape(T, n, vd)
    assert np.abs(got - want).max() <= 1e-6 * np.abs(want).max()


# ---- retention ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H,dk,dv,rot", [(2, 8, 8, 8), (3, 12, 20, 4), (2, 10, 6, 0), (4, 32, 32, 32), (2, 64, 64, 64), (2, 64, 48, 32),
                                         (1, 100, 33, 50), (2, 128, 128, 128), (1, 256, 40, 128), (1, 130, 70, 2), (1, 64, 256, 64)])
def test_retention(dtype, H, dk, dv, rot):
    """Two sequences in one step, then continued in portions and single tokens, with decays from one (nothing is ever lost) to
    one half; a loud pair written at token 3 (and one at 130) that later queries ask for; slots that held rubbish; a slot
    used again."""
    from tinyllama_c_b200.parts.mixers.retention import RetentionMixer
    decay = [1.0, 0.5, 0.999, 0.97][:H] if H > 1 else [0.9995]
    base, eps = 5000.0, 1e-5
    pos_spec = PartSpec("position", "rope_neox", dict(head_dim=dk, theta=base, rope_dim=rot)) if rot else PartSpec("position", "none", dict(head_dim=dk))
    mixer = RetentionMixer(16, H, dk, dv, decay, eps, pos_spec, {n: n for n in "qkvgo"})
    shapes = {s.name: s.shape for s in mixer.weight_specs()}
    mixer.bind({n: torch.zeros(shape) for n, shape in shapes.items()}, DT[dtype], torch.device("cuda"))
    state = torch.full((3, H, dv, dk), 3.0, device="cuda")
    cache = LayerCache(state={mixer.cache_key: state})
    (req,) = mixer.step_requests()

    def call(rows, step):
        y = mixer.mix(dev(rows), step, cache)
        torch.cuda.synchronize()
        return y.float().cpu().numpy().astype(np.float64)

    def make(T, seed):
        r = np.random.default_rng(seed)
        q, k, v, gate = (r.standard_normal((T, H, n)) for n in (dk, dk, dv, dv))
        freq = plain.frequencies(dict(base=base, dims=rot)) if rot else np.zeros(0)
        v *= 0.1
        for loud in (3, 130):
            if loud < T:
                v[loud] = r.standard_normal((H, dv)) * 3.0
                # later queries turned so that they meet the loud key after both rotations
                for t in range(loud + 5, T, 3):
                    q[t] = plain.rotate_halves(k[loud][None], [loud - t], freq)[0] * 0.5 + 0.1 * q[t]
        return np.concatenate([x.reshape(T, -1) for x in (q, k, v, gate)], axis=1).astype(np.float32).astype(np.float64)

    def want_of(rows):
        T = len(rows)
        q, k, v, gate = np.split(rows, np.cumsum([H * dk, H * dk, H * dv]), axis=1)
        freq = plain.frequencies(dict(base=base, dims=rot)) if rot else np.zeros(0)
        q = plain.rotate_halves(q.reshape(T, H, dk), np.arange(T), freq)
        k = plain.rotate_halves(k.reshape(T, H, dk), np.arange(T), freq) * dk ** -0.5
        o = np.stack([plain.retention_scan(q[:, h], k[:, h], v.reshape(T, H, dv)[:, h], decay[h]) for h in range(H)], axis=1)
        return plain.unit_rms(o, eps).reshape(T, -1) * plain.silu(gate), o

    tol = 2e-4 if dtype == "float32" else 8e-3
    step_args = dict(chunk_rows=req.rows, chunk_from=req.from_rows)
    seqs = [make(n, 10 + i) for i, n in enumerate([330, 197])]
    got = run_schedule(seqs, [0, 2], [[203, 1, 1, 61, 64], [90, 1, 1, 3, 102]], call, **step_args)
    for i, s in enumerate(seqs):
        want, o = want_of(s)
        err = np.abs(got[i] - want).max(1)
        assert err.max() <= tol * np.abs(want).max(), f"sequence {i} row {int(err.argmax())}: {err.max():.3e} of {np.abs(want).max():.3e}"
        lost = want_of(np.where(np.arange(len(s))[:, None] == 3, 0.0, s))[1]
        assert np.abs(o[180:] - lost[180:]).max() > 0.05 * np.abs(o[180:]).max()                    # token 3 is still heard
    third = make(70, 33)
    got = run_schedule([third], [0], [[64, 6]], call, **step_args)
    assert np.abs(got[0] - want_of(third)[0]).max() <= tol * np.abs(want_of(third)[0]).max(), "a slot that is used again"
    # the states themselves, and many short sequences that start and go on in one step
    short = [make(n, 50 + n) for n in (2, 40, 65)]
    got = run_schedule(short, [2, 1, 0], [[2], [33, 7], [1, 64]], call, **step_args)
    for i, s in enumerate(short):
        want = want_of(s)[0]
        assert np.abs(got[i] - want).max() <= tol * np.abs(want).max(), f"short sequence {i}"


@pytest.mark.parametrize("H,dk,dv,rot", [(3, 128, 128, 128), (2, 64, 96, 32), (2, 36, 72, 8), (4, 32, 32, 0), (1, 100, 128, 96), (2, 8, 4, 8)])
def test_retention_in_chunks_to_32_bits(H, dk, dv, rot):
    """The chunk kernels with a 32-bit result: pairs of TF32 numbers must give what 32-bit products give.  Two prompts of many
    chunks, one of which goes on (its state and an odd last chunk), a third of a single row."""
    g = np.random.default_rng(dk)
    decay, eps = [0.9995, 1.0, 0.7, 0.98][:H], 1e-5
    freq = plain.frequencies(dict(base=3000.0, dims=rot)) if rot else np.zeros(0)
    state = torch.full((4, H, dv, dk), 5.0, device="cuda")
    width = 2 * H * (dk + dv) + 8
    offs = [4, 4 + H * dk, 4 + 2 * H * dk, 4 + 2 * H * dk + H * dv]
    seqs = [g.standard_normal((n, width)).astype(np.float32).astype(np.float64) for n in (211, 150, 2)]

    def call(rows, step):
        assert ops.retention_chunked_ok(dev(rows), offs, dk, dv, rot, 64)
        out = torch.empty((len(rows), H * dv), device="cuda")
        ops.retention_chunked(dev(rows), *offs, dev(freq), dev(decay), dk ** -0.5, eps, state, step, step.chunks[64], 64, H, dk, dv, out)
        torch.cuda.synchronize()
        return out.cpu().numpy().astype(np.float64)

    got = run_schedule(seqs, [0, 3, 1], [[130, 81], [65, 85], [1, 1]], call, chunk_rows=64, chunk_from=0)
    for i, s in enumerate(seqs):
        T = len(s)
        take = lambda o, n: s[:, o:o + H * n].reshape(T, H, n)
        q = plain.rotate_halves(take(offs[0], dk), np.arange(T), freq)
        k = plain.rotate_halves(take(offs[1], dk), np.arange(T), freq) * dk ** -0.5
        o = np.stack([plain.retention_scan(q[:, h], k[:, h], take(offs[2], dv)[:, h], decay[h]) for h in range(H)], axis=1)
        want = plain.unit_rms(o, eps).reshape(T, -1) * plain.silu(s[:, offs[3]:offs[3] + H * dv])
        err = np.abs(got[i] - want).max(1)
        assert err.max() <= 3e-5 * np.abs(want).max(), f"sequence {i} row {int(err.argmax())}: {err.max():.3e} of {np.abs(want).max():.3e}"


# ---- capped scores without a sink ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H,KV,hd", [(6, 3, 24), (4, 2, 64), (4, 1, 80), (8, 2, 128)])
def test_capped_scores(dtype, H, KV, hd):
    """Prompts (one continues at position 300) and single tokens with one key loud enough that its score meets the cap: alone it
    would take all the weight, capped it does not."""
    g = gen(51)
    cap = 2.5
    starts, lens = [0, 300, 63, 5], [270, 40, 2, 1]
    pos, row_seq, cu, start_pos = _step_arrays(starts, lens)
    totals = [s + n for s, n in zip(starts, lens)]
    slots, table, k_pages, v_pages = _paged_setup(g, 4, totals, KV, hd, DT[dtype])
    for seq, p in ((0, 3), (0, 64), (1, 10), (1, 127)):
        k_pages[int(table[int(slots[seq]), p // 64]), :, p % 64, :] *= 40.0
    T = sum(lens)
    q = rnd(g, T, H * hd, dtype=DT[dtype])
    tol = KTOL[DT[dtype]] * 2.5
    args = [q, k_pages, v_pages, table, pos, row_seq, slots, torch.empty(T, H * hd, dtype=DT[dtype]), H, KV, hd,
            1.0 / math.sqrt(hd), 0, 0, cu, start_pos, max(totals), 0, 0, cap, False]
    cmp("attention", args, [7], tol_of=tol)
    capped = args[7].float().clone()
    ops_plain.attention(*args[:-2], 0.0, False)
    assert (args[7].float() - capped).abs().max() > 0.1 * capped.abs().max()
    starts = [0, 269, 63, 700]
    pos, row_seq, cu, _ = _step_arrays(starts, [1] * 4)
    slots, table, k_pages, v_pages = _paged_setup(g, 4, [s + 1 for s in starts], KV, hd, DT[dtype])
    k_pages[int(table[int(slots[3]), 2]), :, 5, :] *= 40.0
    q = rnd(g, 4, H * hd, dtype=DT[dtype])
    cmp("attention", [q, k_pages, v_pages, table, pos, row_seq, slots, torch.empty(4, H * hd, dtype=DT[dtype]), H, KV, hd,
                      1.0 / math.sqrt(hd), 0, 701, None, None, 0, 0, 0, cap, False], [7], tol_of=tol)


# ---- the polynomial over normed powers ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("F", [1, 5, 320, 500, 2048, 2050, 4096, 9000, 12288, 20003])
def test_polynomial_over_normed_powers(dtype, F):
    g = np.random.default_rng(F)
    T, eps = 7, 1e-5
    z = g.standard_normal((T, F))
    z[1] *= 30.0
    z[2] *= 0.02                                   # eps matters for the square and rules the cube
    z[3, F // 2] = 50.0                            # one loud value
    z = np.concatenate([z, np.ones((T, 4))], axis=1).astype(np.float32)
    tol = 3e-5 if dtype == "float32" else 6e-3
    for coeff in ((1.0, 0.0, 0.0, 0.0), (0.0, 1.0, 0.0, 0.0), (0.0, 0.0, 1.0, 0.0), (0.0, 0.0, 0.0, -0.7), (0.7, -1.3, 0.4, 0.25)):
        out = torch.empty((T, F), dtype=DT[dtype], device="cuda")
        ops.polynorm(dev(z)[:, :F], coeff, eps, out)
        want = plain.polynorm(z[:, :F].astype(np.float64), coeff, eps)
        err = np.abs(out.float().cpu().numpy() - want).max(1)
        assert np.all(err <= tol * np.maximum(np.abs(want).max(1), 1e-3)), f"{coeff}: {err}"

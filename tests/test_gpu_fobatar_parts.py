"""Each Fobatar mechanism alone on the GPU against its plain function (tests/plain/fobatar_plain.py), on inputs made so that a
fault shows: keys of the query's own chunk, a sink of score 0 and a gate per head in all four attention kernels (the warp
kernel, single tokens with the keys split, prompts on tcgen05 with the keys whole and in ranges, single tokens in one
kernel), with one loud key just inside and just outside a chunk's edge, at page borders; the same gate in both latent
kernels; whole mixers over schedules of prompts, portions and single tokens, with a loud row under a loud oldest tap, a key
that decides the output, slots that held rubbish and pages that are over filled with large numbers; the norm over padded
heads; experts chosen by a table, with both clamps at work; the clamped swish in the epilogue of every product kernel; the
embedding added once more; a norm with a multiplier."""
import math

import numpy as np
import pytest
import torch

from tinyllama_c_b200 import ops
from tinyllama_c_b200.cache import Cache
from tinyllama_c_b200.engine.step import StepEntry, pack
from tinyllama_c_b200.parts.base import PartSpec, step_scratch
from plain import ops_plain
from plain import fobatar_plain as plain
from test_gpu_kernels import TOL as KTOL, _paged_setup, _step_arrays, cmp, gen, rnd

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dev(a, dtype=torch.float32):
    return torch.tensor(np.ascontiguousarray(a), dtype=dtype, device="cuda")


# ---- chunks, a sink and a gate per head: the four attention kernels ---------------------------------------------------------------
def _loud_edges(k_pages, table, slots, seq, last, chunk):
    """Makes the last key of the previous chunk and the first key of `last`'s own stand out for every query of `last`."""
    edge = last // chunk * chunk
    for p, f in ((edge - 1, 8.0), (edge, 6.0)):
        if 0 <= p <= last:
            k_pages[int(table[int(slots[seq]), p // 64]), :, p % 64, :] *= f


CHUNKS = [1, 5, 33, 64, 100, 128, 1000]


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("chunk", CHUNKS)
@pytest.mark.parametrize("H,KV,hd", [(6, 3, 24), (4, 1, 80), (9, 1, 64)])
def test_chunks_and_head_gate_of_any_rows_and_of_split_keys(dtype, H, KV, hd, chunk):
    """The warp kernel on a step that mixes prompts (one continues inside a chunk) with single rows, and the split-key kernels of
    single-token steps."""
    g = gen(51)
    starts, lens = [0, 300, 63, 5], [270, 40, 2, 1]
    pos, row_seq, cu, _ = _step_arrays(starts, lens)
    slots, table, k_pages, v_pages = _paged_setup(g, 4, [s + n for s, n in zip(starts, lens)], KV, hd, DT[dtype])
    T = sum(lens)
    q, wide = rnd(g, T, H * hd, dtype=DT[dtype]), rnd(g, T, H + 5, scale=2.0)
    gate = wide[:, 3:3 + H]
    for seq, last in ((0, 269), (0, 128), (1, 339)):
        _loud_edges(k_pages, table, slots, seq, last, chunk)
    args = [q, k_pages, v_pages, table, pos, row_seq, slots, torch.empty(T, H * hd, dtype=DT[dtype]), H, KV, hd,
            1.0 / math.sqrt(hd), 0, 0, None, None, 0, 0, 0, 0.0, True, 0, None, chunk, gate]
    cmp("attention", args, [7], tol_of=KTOL[DT[dtype]] * 2)
    starts = [0, 269, 63, 700, 128]
    pos, row_seq, cu, _ = _step_arrays(starts, [1] * 5)
    slots, table, k_pages, v_pages = _paged_setup(g, 5, [s + 1 for s in starts], KV, hd, DT[dtype], n_slots=6)
    q, gate = rnd(g, 5, H * hd, dtype=DT[dtype]), rnd(g, 5, H, scale=2.0)
    for seq, last in ((1, 269), (3, 700), (4, 128)):
        _loud_edges(k_pages, table, slots, seq, last, chunk)
    for max_keys in (701, 1024):
        cmp("attention", [q, k_pages, v_pages, table, pos, row_seq, slots, torch.empty(5, H * hd, dtype=DT[dtype]), H, KV,
                          hd, 1.0 / math.sqrt(hd), 0, max_keys, None, None, 0, 0, 0, 0.0, True, 0, None, chunk, gate], [7],
            tol_of=KTOL[DT[dtype]] * 2)


@pytest.mark.parametrize("key_ranges", [0, 3])
@pytest.mark.parametrize("chunk", CHUNKS)
@pytest.mark.parametrize("H,KV,hd", [(8, 2, 128), (6, 1, 64), (3, 3, 64)])
def test_chunks_and_head_gate_of_prompts_on_tcgen05(H, KV, hd, chunk, key_ranges):
    """Prompts that cross 128-row tiles and several chunks, one that continues at position 2,100, single rows; the keys whole and
    cut into ranges."""
    g = gen(52)
    starts, lens = [0, 2100, 0, 63, 0], [333, 129, 70, 2, 1]
    pos, row_seq, cu, start_pos = _step_arrays(starts, lens)
    totals = [s + n for s, n in zip(starts, lens)]
    slots, table, k_pages, v_pages = _paged_setup(g, 5, totals, KV, hd, torch.bfloat16, n_slots=7)
    T = sum(lens)
    q, gate = rnd(g, T, H * hd, dtype=torch.bfloat16), rnd(g, T, H, scale=2.0)
    for seq, last in ((0, 127), (0, 128), (0, 200), (0, 332), (1, 2100), (1, 2163), (1, 2228)):
        _loud_edges(k_pages, table, slots, seq, last, chunk)
    args = [q, k_pages, v_pages, table, pos, row_seq, slots, torch.empty(T, H * hd, dtype=torch.bfloat16), H, KV, hd,
            1.0 / math.sqrt(hd), 0, 0, cu, start_pos, max(totals), 0, key_ranges, 0.0, True, 0, None, chunk, gate]
    cmp("attention", args, [7], tol_of=KTOL[torch.bfloat16] * 2.5)
    torch.cuda.synchronize()
    ops.check_errors()
    if chunk in (33, 100):                             # a chunk one position longer differs by far more
        right = args[7].float().clone()
        ops_plain.attention(*args[:-2], chunk + 1, gate)
        assert (args[7].float() - right).abs().max() > 0.1 * right.abs().max()


@pytest.mark.parametrize("chunk", CHUNKS)
@pytest.mark.parametrize("H,KV,hd,rope", [(8, 2, 128, 64), (6, 1, 64, 64), (4, 4, 64, 0), (2, 2, 256, 128)])
def test_chunks_and_head_gate_of_single_tokens_in_one_kernel(H, KV, hd, rope, chunk):
    """Rotation, store of the new row and attention in one launch: the keys in one piece a block, in several pieces that another
    block merges, and pieces of two rounds."""
    g = gen(53)
    starts = [0, 200, 63, 3300, 127, 128]
    B = len(starts)
    pos, row_seq, cu, _ = _step_arrays(starts, [1] * B)
    slots, table, k_pages, v_pages = _paged_setup(g, B, [s + 1 for s in starts], KV, hd, torch.bfloat16, n_slots=7)
    for seq, last in ((3, 3300), (1, 200), (4, 127), (5, 128)):
        _loud_edges(k_pages, table, slots, seq, last, chunk)
    qkv, gate = rnd(g, B, (H + 2 * KV) * hd), rnd(g, B, H, scale=2.0)
    inv = (1.0 / torch.pow(torch.tensor(1e4, dtype=torch.float64),
                           torch.arange(rope // 2, dtype=torch.float64) * 2 / max(rope, 1))).float()
    scale = 1.3 / math.sqrt(hd)
    k_ref, v_ref = k_pages.clone(), v_pages.clone()
    q_ref = torch.empty(B, H * hd, dtype=torch.bfloat16)
    ops_plain.rope_kv_store(qkv, 0, H * hd, (H + KV) * hd, q_ref, k_ref, v_ref, inv, pos, row_seq, slots, table, H, KV, hd, True)
    out_ref = torch.empty(B, H * hd, dtype=torch.bfloat16)
    ops_plain.attention(q_ref, k_ref, v_ref, table, pos, row_seq, slots, out_ref, H, KV, hd, scale, 0, 0, None, None, 0, 0, 0,
                        0.0, True, 0, None, chunk, gate)
    counters = ops.new_arrival_counters("cuda")
    try:
        for max_keys, passes in ((3301, 0), (4096, 1), (4096, 2), (3301, 1000)):
            ops.attention_decode_fused_passes(passes)
            out = torch.empty(B, H * hd, dtype=torch.bfloat16, device="cuda")
            ops.attention_decode_fused(qkv.cuda(), 0, H * hd, (H + KV) * hd, k_pages.cuda(), v_pages.cuda(), inv.cuda(), True, table.cuda(),
                                       pos.cuda(), row_seq.cuda(), slots.cuda(), out, H, KV, hd, scale, 0, max_keys, counters, 0.0,
                                       True, 0, None, chunk, gate.cuda())
            torch.cuda.synchronize()
            ops.check_errors()
            ref = out_ref.double()
            err = (ref - out.cpu().double()).abs().max()
            assert err <= KTOL[torch.bfloat16] * 2.5 * ref.abs().max(), f"max_keys {max_keys}, passes {passes}: {err}"
    finally:
        ops.attention_decode_fused_passes(0)


def test_a_sink_of_score_zero_and_a_gate_show():
    """One key of score s, a value of one: the output is e^s / (1 + e^s) times the gate's sigmoid."""
    for s, z in ((0.0, 0.0), (-3.0, 2.0), (4.0, -1.5)):
        k_pages, v_pages = torch.full((1, 1, 64, 8), s / 8.0), torch.ones(1, 1, 64, 8)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32).cuda()
        out = torch.empty(1, 8, device="cuda")
        ops.attention(torch.ones(1, 8).cuda(), k_pages.cuda(), v_pages.cuda(), i32([[0]]), i32([0]), i32([0]), i32([0]), out, 1, 1, 8, 1.0,
                      sink=True, chunk=7, head_gate=torch.tensor([[z]]).cuda())
        want = math.exp(s) / (1 + math.exp(s)) / (1 + math.exp(-z))
        assert abs(float(out[0, 0]) - want) < 1e-6


# ---- the whole query and key projections normed over padded heads ------------------------------------------------------------------
@pytest.mark.parametrize("H,KV,dim,stride", [(4, 2, 24, 24), (3, 1, 10, 16), (16, 4, 128, 128), (5, 5, 40, 64)])
def test_whole_projection_norm_of_padded_heads(H, KV, dim, stride):
    g = np.random.default_rng(6)
    T, eps = 7, 1e-5
    q, k = g.standard_normal((T, H, dim)) * 3.0, g.standard_normal((T, KV, dim)) * 1e-3       # (keys so small that eps matters)
    wq, wk = 1 + 0.3 * g.standard_normal((H, dim)), 1 + 0.3 * g.standard_normal((KV, dim))
    pad = lambda a: np.concatenate([a, np.zeros(a.shape[:-1] + (stride - dim,))], axis=-1).reshape(a.shape[:-2] + (-1,))
    buf = dev(np.concatenate([pad(q), pad(k), np.full((T, 5), 9.0)], axis=1))
    ops.qk_whole_norm(buf, 0, H * stride, dev(pad(wq)), H * stride, KV * stride, dev(pad(wk)), eps, H * dim, KV * dim)
    got = buf.cpu().numpy()
    for a, w, n, off in ((q, wq, H, 0), (k, wk, KV, H * stride)):
        want = plain.rms_norm(a.reshape(T, n * dim).astype(np.float32).astype(np.float64), w.reshape(-1), eps).reshape(T, n, dim)
        have = got[:, off:off + n * stride].reshape(T, n, stride)
        assert np.abs(have[..., :dim] - want).max() <= 2e-5 * np.abs(want).max() and not have[..., dim:].any()
    assert np.all(got[:, -5:] == 9.0)


# ---- whole mixers -----------------------------------------------------------------------------------------------------------------
# sizes of portions per sequence: whole prompts; portions down to one token; single tokens from the start; a prompt, then single
# tokens across page and chunk borders
SCHEDULES = [([200, 9, 1], [[200], [9], [1]]), ([150, 97], [[17, 1, 2, 1, 99, 30], [64, 1, 3, 20, 9]]), ([40, 12], [[1] * 40, [1] * 12]),
             ([150, 70], [[90] + [1] * 60, [66] + [1] * 4]), ([30, 7], [[2] * 15, [1, 2, 2, 2]])]


def run_mixer(mixer, seqs, cuts, dtype, poison=False):
    """seqs: arrays [T, D] of normed inputs; cuts: the sizes of every sequence's portions.  Drives the mixer through the library's
    cache in slots that held rubbish; poison: pages that the cache has given back are filled with a large number after
    every step.  Returns the outputs per sequence."""
    cache = Cache({0: mixer.cache_requests()}, max_tokens=64 * 16, max_seqs=len(seqs) + 2, dtype=DT[dtype], device="cuda")
    for grp in cache.state_groups:
        grp.data.fill_(7.0)
    slots = [cache.acquire() for _ in range(len(seqs) + 1)][1:]          # (slot 0 stays unused)
    outs, at = [[] for _ in seqs], [0] * len(seqs)
    for s in range(max(len(c) for c in cuts)):
        live = [i for i in range(len(seqs)) if s < len(cuts[i])]
        entries = [StepEntry(slots[i], [0] * cuts[i][s]) for i in live]
        starts = [cache.reserve(e.slot, len(e.tokens)) for e in entries]
        step, _, _ = pack(entries, starts, 1, torch.device("cuda"))
        cache.upload_tables()
        rows = dev(np.concatenate([seqs[i][at[i]:at[i] + cuts[i][s]] for i in live]), DT[dtype])
        out = torch.full((step.n_rows, mixer.hidden), 3.0, device="cuda")
        with step_scratch(step):
            mixer.forward(rows, step, cache.layer_view(0), out, accumulate=False)
        y, o = out.cpu().numpy().astype(np.float64), 0
        for i in live:
            outs[i].append(y[o:o + cuts[i][s]])
            at[i] += cuts[i][s]
            o += cuts[i][s]
            cache.commit(slots[i], cuts[i][s])
        if poison:
            for grp in cache.kv_groups:
                free = [p for p in range(grp.pool.n) if p not in set(grp.pool.held())]
                if free:
                    grp.k[:, free] = 1e4
                    if grp.v is not None:
                        grp.v[:, free] = 1e4
    cache.check()
    ops.check_errors()
    return [np.concatenate(x) for x in outs]


def _bind(part, W, dtype):
    part.bind({k: torch.tensor(v, dtype=torch.float32).to(torch.bfloat16) for k, v in W.items()}, DT[dtype], torch.device("cuda"))
    return part


def _round_all(W):
    return {k: plain.bf16_round(v) for k, v in W.items()}


RAMP = dict(factor=4.0, original=64, fast=8.0, slow=1.0)


@pytest.mark.parametrize("at_once", [True, False])
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H,KV,dim,vdim,taps,rot,chunk", [
    (4, 2, 24, 16, 3, dict(base=100.0, dims=8, scaling=RAMP), 37), (3, 1, 16, 20, 1, dict(base=5000.0, dims=16), 5),
    (4, 2, 64, 64, 4, dict(base=10000.0, dims=32, scaling=RAMP), 100), (2, 2, 128, 128, 2, dict(base=700.0, dims=128, scaling=RAMP), 64),
    (6, 2, 64, 48, 5, dict(base=700.0, dims=0), None), (3, 3, 40, 64, 4, dict(base=900.0, dims=20, scaling=RAMP), 150),
    (9, 1, 128, 64, 4, dict(base=900.0, dims=6), 33)])
def test_chunked_attention_mixer_over_schedules(monkeypatch, dtype, H, KV, dim, vdim, taps, rot, chunk, at_once):
    """The whole mixer, with convolution, norm, rotation and stores in one kernel and in kernels of their own: the oldest tap speaks loudest and one row is loud, so an echo one row short or long shows; the sharp
    score scale makes single keys decide."""
    monkeypatch.setattr(ops, "DISABLE_QKV_PREPARE", not at_once)
    D, eps = 40, 1e-5
    g = np.random.default_rng(H * 100 + dim)
    W = {"q": g.standard_normal((H * dim, D)), "k": g.standard_normal((KV * dim, D)), "v": g.standard_normal((KV * vdim, D)),
         "g": g.standard_normal((H, D)), "o": g.standard_normal((D, H * vdim))}
    W = {n: w / math.sqrt(w.shape[1]) for n, w in W.items()}
    for n, c in (("q", H * dim), ("k", KV * dim), ("v", KV * vdim)):
        W[n + ".conv"] = g.standard_normal((c, taps)) * np.linspace(2.0, 0.5, taps)[None, :]
    W["q.norm"], W["k.norm"] = 1 + 0.3 * g.standard_normal(H * dim), 1 + 0.3 * g.standard_normal(KV * dim)
    W = _round_all(W)
    m = dict(heads=H, kv_heads=KV, dim=dim, vdim=vdim, conv=taps, scale=2.0 / math.sqrt(dim), rot=rot)
    if chunk:
        m["mask"] = dict(size=chunk)
    pos = PartSpec("position", "rope_interleaved", dict(head_dim=dim, theta=rot["base"], rope_dim=rot["dims"],
                                                        scaling=dict(rot["scaling"], kind="ramp") if "scaling" in rot else None)) \
        if rot["dims"] else PartSpec("position", "none", dict(head_dim=dim))
    mixer = _bind(PartSpec("mixer", "attention", dict(
        hidden=D, n_heads=H, n_kv_heads=KV, head_dim=dim, v_dim=vdim, prefix="", position=pos, scale=m["scale"], conv_taps=taps,
        names={k: k for k in "qkvgo"}, whole_norm=dict(q="q.norm", k="k.norm", eps=eps), sink=True, chunk=chunk, gate="sigmoid",
        gate_per="head")).build(), W, dtype)
    for lens, cuts in SCHEDULES:
        seqs = [plain.bf16_round(g.standard_normal((n, D))) for n in lens]
        seqs[0][min(20, lens[0] - 1)] *= 6.0
        got = run_mixer(mixer, seqs, cuts, dtype, poison=True)
        for x, y in zip(seqs, got):
            want = plain.chunked_attention(x, W, "", m, eps)
            if dtype == "float32":
                assert np.abs(y - want).max() <= 1e-4 * np.abs(want).max(), f"portions {cuts[0][:4]}"
            else:
                noise = np.sqrt(((plain.chunked_attention(x, W, "", m, eps, plain.bf16_round) - want) ** 2).mean(1)).max()
                err = np.sqrt(((y - want) ** 2).mean(1))
                assert err.max() <= 3.0 * noise, f"portions {cuts[0][:4]}: {err.max():.2e} at row {err.argmax()}, noise {noise:.2e}"


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H,dim,r,vdim,R,rot", [
    (3, 10, 6, 14, 20, dict(base=100.0, dims=4, scaling=RAMP)), (5, 16, 16, 24, 48, dict(base=10000.0, dims=16, scaling=RAMP)),
    (2, 32, 32, 16, 128, dict(base=700.0, dims=32)), (17, 8, 16, 8, 144, dict(base=900.0, dims=12, scaling=RAMP)),
    (1, 4, 2, 4, 8, dict(base=50.0, dims=2, scaling=RAMP))])
def test_latent_attention_mixer_over_schedules(dtype, H, dim, r, vdim, R, rot):
    """The whole mixer with a ramp and enlarged cosines and sines on the rotated part only, no sink, a gate per head; a sharp
    score scale, and one token whose key stands out for the tokens after it."""
    D, eps = 40, 1e-5
    g = np.random.default_rng(H * 100 + R)
    W = {"q": g.standard_normal((H * (dim + r), D)), "dkv": g.standard_normal((R + r, D)), "uk": g.standard_normal((H * dim, R)),
         "uv": g.standard_normal((H * vdim, R)), "g": g.standard_normal((H, D)), "o": g.standard_normal((D, H * vdim))}
    W = {n: w / math.sqrt(w.shape[1]) for n, w in W.items()}
    W["dkv.norm"] = 1 + 0.3 * g.standard_normal(R)
    W = _round_all(W)
    m = dict(heads=H, dim=dim, rot_dim=r, vdim=vdim, kv_rank=R, scale=2.0 / math.sqrt(dim + r), rot=rot)
    pos = PartSpec("position", "rope_interleaved", dict(head_dim=r, theta=rot["base"], rope_dim=rot["dims"],
                                                        scaling=dict(rot["scaling"], kind="ramp") if "scaling" in rot else None))
    mixer = _bind(PartSpec("mixer", "latent_attention", dict(
        hidden=D, n_heads=H, head_dim=dim, rot_dim=r, v_dim=vdim, kv_rank=R, scale=m["scale"], eps=eps, position=pos,
        names=dict({k: k for k in ("q", "dkv", "uk", "uv", "g", "o")}, dkv_norm="dkv.norm"))).build(), W, dtype)
    for lens, cuts in SCHEDULES:
        seqs = [plain.bf16_round(g.standard_normal((n, D))) for n in lens]
        seqs[0][min(3, lens[0] - 1)] *= 4.0
        got = run_mixer(mixer, seqs, cuts, dtype)
        for x, y in zip(seqs, got):
            want = plain.latent_attention(x, W, "", m, eps)
            if dtype == "float32":
                assert np.abs(y - want).max() <= 1e-4 * np.abs(want).max(), f"portions {cuts[0][:4]}"
            else:
                noise = np.sqrt(((plain.latent_attention(x, W, "", m, eps, plain.bf16_round) - want) ** 2).mean(1)).max()
                err = np.sqrt(((y - want) ** 2).mean(1))
                assert err.max() <= 4.0 * noise, f"portions {cuts[0][:4]}: {err.max():.2e} at row {err.argmax()}, noise {noise:.2e}"


# ---- experts chosen by a table --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("V,E,top,T", [(50, 4, 2, 1), (50, 4, 4, 33), (1000, 40, 3, 300), (7, 1, 1, 9), (300, 100, 7, 2049), (90, 32, 5, 500)])
def test_routing_by_a_table(V, E, top, T):
    g = np.random.default_rng(E)
    table = np.stack([g.permutation(E)[:top] for _ in range(V)]).astype(np.int32)
    toks = g.integers(0, V, T).astype(np.int32)
    for tile in (32, 64):
        # between two other tables: every one of a launch has ranges of its own
        others = [(dev(table[:, :1], torch.int32), E, False), (dev(np.tile(np.arange(2), (V, 1)), torch.int32), 2, True)]
        tables = ops.ExpertTables([others[0], (dev(table, torch.int32), E, tile == 64), others[1]])
        tile = 64 if tile == 64 and T * top >= 64 * E else 32
        routed = ops.moe_route_tables(dev(toks, torch.int32), tables)
        assert np.array_equal(routed[0][0].cpu().numpy(), table[toks][:, 0]) and np.array_equal(routed[2][0].cpu().numpy(), np.tile([0, 1], T))
        ids, wts, order, offsets, tile_off, rows = routed[1]
        want = table[toks].reshape(-1)
        assert np.array_equal(ids.cpu().numpy(), want) and rows == tile
        assert np.allclose(wts.cpu().numpy(), 1.0 / top)
        order, offsets, tile_off = order.cpu().numpy(), offsets.cpu().numpy(), tile_off.cpu().numpy()
        counts = np.bincount(want, minlength=E)
        assert np.array_equal(offsets, np.concatenate([[0], np.cumsum(counts)]))
        assert np.array_equal(tile_off, np.concatenate([[0], np.cumsum((counts + tile - 1) // tile)]))
        assert np.array_equal(np.sort(order), np.arange(T * top)) and np.array_equal(want[order], np.repeat(np.arange(E), counts))


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("D,F,E,top,shared", [(40, 24, 5, 2, (16, 0.5)), (52, 20, 3, 3, (12, 2.0)), (64, 96, 8, 3, None), (64, 40, 1, 1, (96, 1.0)),
                                              (64, 24, 40, 4, (24, 0.3))])
def test_experts_of_a_table_with_both_clamps_at_work(dtype, D, F, E, top, shared):
    g = np.random.default_rng(D + F + E)
    V, p = 30, "m."
    W = {f"{p}e{e}.{n}": g.standard_normal(s) / math.sqrt(s[1]) for e in range(E) for n, s in (("gate", (F, D)), ("up", (F, D)), ("down", (D, F)))}
    mlp = dict(router=dict(experts=E, top=top), expert=dict(ff=F, limit=0.8))
    part = None
    if shared:
        Fs, lim = shared
        mlp["shared"] = dict(ff=Fs, limit=lim)
        W.update({f"{p}shared.{n}": g.standard_normal(s) / math.sqrt(s[1]) for n, s in (("gate", (Fs, D)), ("up", (Fs, D)), ("down", (D, Fs)))})
        part = PartSpec("feed_forward", "swiglu", dict(hidden=D, intermediate=Fs, prefix=p + "shared.", names=dict(gate="gate", up="up", down="down"),
                                                       act="swish_clamped", limit=lim, alpha=1.702))
    W = _round_all(W)
    W[p + "table"] = np.stack([g.permutation(E)[:top] for _ in range(V)])
    ff = PartSpec("feed_forward", "moe", dict(
        hidden=D, n_experts=E, top=top, expert_ff=F, router_name=None, table_name=p + "table", vocab=V,
        expert_names={k: p + "e{e}." + k for k in ("gate", "up", "down")}, weight_on="output", act="swish_clamped", limit=0.8, alpha=1.702,
        shared=part)).build()
    tensors = {k: torch.tensor(v, dtype=torch.int32) if k.endswith("table") else torch.tensor(v, dtype=torch.float32).to(torch.bfloat16)
               for k, v in W.items()}
    ff.bind(tensors, DT[dtype], torch.device("cuda"))
    for T in (1, 5, 40, 130, 400):
        x, toks = plain.bf16_round(g.standard_normal((T, D)) * 2.0), g.integers(0, V, T)
        out = torch.full((T, D), 5.0, device="cuda")
        step = type("Step", (), dict(tokens=dev(toks, torch.int32), scratch={}))
        ff.forward(dev(x, DT[dtype]), out, accumulate=False, step=step)
        want = plain.table_moe(x, toks, W, p, mlp)
        tol = 3e-5 if dtype == "float32" else 1.2e-2
        assert np.abs(out.cpu().numpy() - want).max() <= tol * np.abs(want).max(), f"{T} rows"
        before = out.clone()
        ff.route_step([ff], ops.ExpertTables([ff.table_entry()]), step)       # the routing made ahead of the layers is the same
        out.fill_(5.0)
        ff.forward(dev(x, DT[dtype]), out, accumulate=False, step=step)
        assert torch.equal(before, out)
    with pytest.raises(ValueError, match="token ids"):
        ff.forward(dev(x, DT[dtype]), out)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("M", [1, 8, 20, 33, 64, 100, 300])
@pytest.mark.parametrize("F,K", [(8, 40), (96, 64), (1000, 264), (2048, 512)])
def test_clamped_swish_in_the_products_epilogue(dtype, M, F, K):
    """Gate and up values on both sides of the limits, in every product kernel (by the number of rows and the output's width)."""
    g = gen(55)
    a, w = rnd(g, M, K, dtype=DT[dtype]), rnd(g, 2 * F, K, dtype=DT[dtype], scale=2.0 / math.sqrt(K))
    for limit, alpha in ((0.9, 1.702), (0.2, 1.0)):
        cmp("linear_swiglu", [a, w, torch.empty(M, F, dtype=DT[dtype]), None, None, "swish_clamped", limit, alpha], [2], tol_of=KTOL[DT[dtype]] * 2)
    ops.check_errors()


# ---- the embedding once more, a norm with a multiplier ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("D", [5, 52, 64, 2048])
def test_embedding_added_to_the_stream(dtype, D):
    g = np.random.default_rng(9)
    table, x = plain.bf16_round(g.standard_normal((40, D))), g.standard_normal((33, D)).astype(np.float32)
    toks = g.integers(0, 40, 33)
    xd, first = dev(x), torch.empty((33, D), device="cuda")
    ops.embed_add(dev(toks, torch.int32), dev(table, DT[dtype]), 1.7, xd)
    want = x.astype(np.float64) + table[toks] * 1.7
    assert np.abs(xd.cpu().numpy() - want).max() <= 1e-6 * np.abs(want).max()
    ops.embed(dev(toks, torch.int32), dev(table, DT[dtype]), 1.7, first)
    assert np.abs(first.cpu().numpy() - table[toks] * 1.7).max() <= 1e-6 * np.abs(table).max()


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("D,T", [(5, 3), (52, 9), (64, 300), (2048, 8), (2048, 1500), (4098, 4)])
def test_output_norm_that_leaves_the_next_norm_of_the_stream(dtype, D, T):
    """One kernel adds a normed result (a sum of terms) into the stream and norms the new rows for the sublayer that follows."""
    g = np.random.default_rng(D)
    w, w2 = 1 + 0.2 * g.standard_normal(D), 1 + 0.2 * g.standard_normal(D)
    parts, extra, x = g.standard_normal((T, 3, D)), g.standard_normal((T, D)), g.standard_normal((T, D)) * 0.01
    make = lambda name, weight, scale: PartSpec("norm", "rmsnorm", dict(width=D, eps=1e-5, weight_name=name, scale=scale)).build()
    norm, nxt = make("w", w, 0.003), make("v", w2, 1.0)                # (a stream so small that eps matters)
    for n, v in ((norm, w), (nxt, w2)):
        n.bind({"w": torch.tensor(v), "v": torch.tensor(v)}, torch.float32, torch.device("cuda"))
    xd, left = dev(x), torch.full((T, D), 7.0, dtype=DT[dtype], device="cuda")
    norm.add_normed(dev(parts), xd, dev(extra), None, copy=left, next_norm=nxt)
    want = x + 0.003 * plain.rms_norm(parts.sum(1) + extra, w, 1e-5)
    assert np.abs(xd.cpu().numpy() - want).max() <= 2e-5 * np.abs(want).max()
    want = plain.rms_norm(want, w2, 1e-5)
    assert np.abs(left.float().cpu().numpy() - want).max() <= (3e-5 if dtype == "float32" else 5e-3) * np.abs(want).max()


def test_norm_with_a_multiplier_adds_into_the_stream():
    g = np.random.default_rng(10)
    w, y, x = 1 + 0.2 * g.standard_normal(52), g.standard_normal((9, 52)) * 3.0, g.standard_normal((9, 52))
    norm = PartSpec("norm", "rmsnorm", dict(width=52, eps=1e-5, weight_name="w", scale=0.3)).build()
    norm.bind({"w": torch.tensor(w)}, torch.float32, torch.device("cuda"))
    xd = dev(x)
    norm.add_normed(dev(y), xd)
    want = x + 0.3 * plain.rms_norm(y, w, 1e-5)
    assert np.abs(xd.cpu().numpy() - want).max() <= 1e-5 * np.abs(want).max()

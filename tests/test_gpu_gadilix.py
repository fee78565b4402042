"""GPU tests of the Gadilix stack against the plain float64 restatement in gadilix_ref.py, on small random models made here.

Gates: with gpt.compute_dtype = float32 the logits agree to 2e-4 (rms of the difference, mean removed, over the rms of the logits);
in bf16 nine rows in ten to 6e-2.  Weights are drawn on the bf16 grid, so both sides hold the same numbers.  Where random weights would
hide a fault they are shaped: the norm weights of the queries scaled up so that the softmax is peaked (a window or block edge one position
off, a mean row of the wrong block, a lost far block then moves the logits far -- each such test shows that on the oracle first).
"""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import koifish_b200 as kf
import gadilix_ref as ref
from gadilix_models import attn, bf16_grid, bits, config, layer, moe, set_all, st_entries, tokens, weights
from st_util import write_safetensors

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {True: 2e-4, False: 6e-2}


@pytest.fixture(scope="module")
def ctx():
    c = kf.Context(0)
    yield c
    c.close()


def build(ctx, cfg, W, f32, max_seq=256, slots=2, panel=64, logit_rows=None):
    gpt = {"max_seq_len": max_seq, "max_batch": slots, "max_prefill": panel, "logit_rows": logit_rows or panel}
    if f32:
        gpt["compute_dtype"] = "float32"
    m = kf.Model(ctx, {"hf_config": cfg, "gpt": gpt})
    assert sorted(m.tensor_names()) == sorted(W.keys())
    set_all(m, W)
    return m


def rel(got, want, q=1.0):
    """largest (q = 1) or q-quantile row error: rms of the difference, mean removed, over the rms of the wanted logits"""
    d = np.asarray(got, dtype=np.float64) - np.asarray(want, dtype=np.float64)
    d = d - d.mean(-1, keepdims=True)
    w = np.asarray(want, dtype=np.float64)
    w = w - w.mean(-1, keepdims=True)
    return float(np.quantile(np.atleast_1d(np.sqrt((d ** 2).mean(-1))), q) / np.sqrt((w ** 2).mean()))


def close(got, want, f32):
    if f32:
        return rel(got, want) < TOL[True]
    return rel(got, want, 0.9) < TOL[False] and rel(got, want) < 0.5


def oracle(cfg, W, toks):
    return ref.forward(cfg, W, list(toks)).numpy()


def run_cut(model, toks, cuts, slot=0):
    """feed toks in portions of the given sizes (the rest one by one); fp32 logits of every position"""
    out, at = [], 0
    sizes = list(cuts)
    while at < len(toks):
        n = sizes.pop(0) if sizes else 1
        n = min(n, len(toks) - at)
        lg, _ = model.forward_rows(toks[at:at + n], at, slot=slot, rows=list(range(n)))
        out.append(lg)
        at += n
    return np.concatenate(out)


def edited(cfg, fn, i=0):
    """a copy of cfg whose layer i went through fn"""
    c = json.loads(json.dumps(cfg))
    fn(c["layers"][i])
    return c


# five layers, two of them on the tensors of earlier ones
FULL = [layer(attn(), moe()),
        layer(attn(heads=6, kv_heads=3, dim=16, vdim=8, window=21, pool=5), moe(experts=5, top=1, ff=10, shared=8)),
        layer(attn(), moe(), weights_of=0),
        layer(attn(heads=3, kv_heads=3, dim=9, vdim=11, window=6, pool=11), None),
        layer(attn(heads=6, kv_heads=3, dim=16, vdim=8, window=21, pool=5), moe(experts=5, top=1, ff=10, shared=8), weights_of=1)]


# ------------------------------------------------------------------------------------------------------------ each mechanism alone
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("ly", [
    layer(attn()),                                                        # grouped heads, value size != key size
    layer(attn(heads=3, kv_heads=3, dim=8, vdim=8, window=1, pool=1)),    # the token itself and every earlier one as a block
    layer(attn(heads=1, kv_heads=1, dim=70, vdim=33, window=5, pool=2)),  # one wide head, odd values
    layer(attn(window=4, pool=10)),                                       # blocks longer than the window
    layer(attn(window=12, pool=0)),                                       # a window without blocks
    layer(attn(window=0)),                                                # every earlier position
    layer(attn(window=1000, pool=3)),                                     # a window longer than the model's context
    layer(attn(window=7, pool=1000)),                                     # a block longer than the model's context
    layer(attn(heads=8, kv_heads=1, dim=16, vdim=24, window=11, pool=3, scale=0.7)),   # one kv head, a scale of its own
    layer(attn(), moe()),
    layer(attn(), moe(shared=0)),                                         # no shared expert
    layer(attn(), moe(experts=7, top=7, ff=5, shared=9)),                 # every expert of every token
    layer(attn(), moe(experts=1, top=1, ff=24, shared=7)),                # one expert
    layer(attn(), moe(experts=40, top=3, ff=8, shared=12)),               # more experts than lanes
], ids=["attn", "window1_pool1", "one_head", "pool_longer", "no_pool", "all", "long_window", "long_pool", "one_kv_head", "moe", "moe_no_shared", "moe_all",
        "moe_one", "moe_40"])
def test_single_layer_prompt(ctx, ly, f32):
    cfg = config([ly], width=32)
    W = weights(cfg, seed=3, q_gain=2.0)
    toks = tokens(47, cfg["vocab"], 1)
    want = oracle(cfg, W, toks)
    m = build(ctx, cfg, W, f32)
    assert close(run_cut(m, toks, [47]), want, f32)
    assert close(run_cut(m, toks, [9, 2, 13], slot=1), want, f32)
    m.close()


def test_norm_numbers_and_residual_factor(ctx):
    """norm weights (one number each) far from 1 and a residual factor that is no power of two: a norm without its weight, a factor on the
    wrong term or an embedding that is not normed shows"""
    cfg = config([layer(attn(), moe()), layer(attn(), None)], width=32, mult=0.37, eps=3e-3)
    W = weights(cfg, seed=4)
    for k, v in (("embed.norm", 0.07), ("final.norm", -1.75), ("l0.norm1", 2.5), ("l0.norm2", -0.6), ("l1.norm1", 1.4)):
        W[k] = bf16_grid(torch.tensor(v))
    toks = tokens(20, cfg["vocab"], 2)
    want = oracle(cfg, W, toks)
    for alt in (dict(cfg, residual_mult=0.4), dict(cfg, norm={"eps": 1e-5})):
        assert rel(oracle(alt, W, toks), want) > 10 * TOL[True]
    m = build(ctx, cfg, W, True)
    assert rel(run_cut(m, toks, [9, 2]), want) < TOL[True]
    m.close()
    one = dict(cfg)
    one.pop("residual_mult")  # left out: 1
    m = build(ctx, one, W, True)
    assert rel(run_cut(m, toks, [9, 2]), oracle(one, W, toks)) < TOL[True]
    m.close()


def test_shift_is_part_of_the_state(ctx):
    """a shift near 1 -- the mixer reads the previous token almost alone -- cut everywhere, in every layer; the state of a slot that ended is
    not seen by the request that takes the slot"""
    cfg = config([layer(attn(window=5, pool=0), None), layer(attn(), moe()), layer(attn(), moe(), weights_of=1)], width=40)
    W = weights(cfg, seed=5)
    for k in ("l0.shift", "l1.shift"):
        W[k] = bf16_grid(0.9 + 0.2 * W[k])
    toks = tokens(30, cfg["vocab"], 3)
    want = oracle(cfg, W, toks)
    assert rel(oracle(cfg, dict(W, **{"l1.shift": W["l1.shift"] * 0}), toks), want) > 100 * TOL[True]
    m = build(ctx, cfg, W, True)
    for cuts in ([30], [1] * 30, [2] * 15, [5, 1, 17, 7], [29, 1]):
        assert rel(run_cut(m, toks, cuts), want) < TOL[True], cuts
    m.close()


def test_layers_on_shared_tensors(ctx):
    """chains of references, forwards and backwards, each layer with a cache and a shift state of its own"""
    a, b = layer(attn(), moe()), layer(attn(window=6, pool=3), moe(top=1))
    cfg = config([dict(b, weights_of=3), a, dict(a, weights_of=1), b, dict(a, weights_of=2), dict(b, weights_of=0)], width=32)
    W = weights(cfg, seed=7)
    assert set(k.split(".")[0] for k in W) == {"embed", "head", "final", "l1", "l3"}
    toks = tokens(45, cfg["vocab"], 4)
    want = oracle(cfg, W, toks)
    m = build(ctx, cfg, W, True)
    assert rel(run_cut(m, toks, [45]), want) < TOL[True]
    assert rel(run_cut(m, toks, [9, 2, 13]), want) < TOL[True]
    m.close()


# ------------------------------------------------------------------------------------------------------------ whole stacks
@pytest.mark.parametrize("f32", [True, False])
def test_stack_prompt_and_decode(ctx, f32):
    """a prompt in one step, then token by token: both equal the oracle; the first tokens of a sequence decoded one by one as well"""
    cfg = config(FULL)
    W = weights(cfg, seed=5)
    toks = tokens(90, cfg["vocab"], 2)
    want = oracle(cfg, W, toks)
    m = build(ctx, cfg, W, f32)
    assert close(run_cut(m, toks, [64, 26]), want, f32)          # two panels
    assert close(run_cut(m, toks, [50]), want, f32)              # 50 at once, 40 decoded (graph replay from the second step on)
    assert close(run_cut(m, toks[:40], []), want[:40], f32)       # from the very first token one by one
    m.close()


@pytest.mark.parametrize("f32", [True, False])
def test_wide_panels_and_tuned_matmul_widths(ctx, f32):
    """width 128, extents that are multiples of 16, panels of up to 192 tokens: in bf16 the projections run on the tensor-core kernels, the
    dispatch tables of 192 x 4 entries take the many-token form"""
    cfg = config([layer(attn(heads=4, kv_heads=2, dim=32, vdim=32, window=70, pool=8), moe(experts=8, top=4, ff=64, shared=128)),
                  layer(attn(heads=4, kv_heads=4, dim=64, vdim=64, window=33, pool=12), moe(experts=16, top=2, ff=32, shared=48))], width=128, vocab=160)
    W = weights(cfg, seed=14)
    toks = tokens(230, cfg["vocab"], 15)
    want = oracle(cfg, W, toks)
    m = build(ctx, cfg, W, f32, panel=192, logit_rows=192)
    assert close(run_cut(m, toks, [192, 17, 2]), want, f32)
    m.close()


def test_portions_of_many_sizes(ctx):
    cfg = config(FULL)
    W = weights(cfg, seed=6, q_gain=3.0)
    toks = tokens(131, cfg["vocab"], 3)
    want = oracle(cfg, W, toks)
    m = build(ctx, cfg, W, True)
    for cuts in ([2, 2, 3, 2, 64, 2, 31, 2, 17], [1, 2, 1, 63, 64, 1], [7] * 19, [64, 64, 2], [3, 1, 1, 2, 5, 64, 2, 2, 2, 40], [2] * 66):
        assert rel(run_cut(m, toks, cuts), want) < TOL[True], cuts
    m.close()


def test_slots_reused_and_interleaved(ctx):
    """two requests advance alternately in two slots; a released slot is taken by a new request and nothing of the old one shows: not its
    rows, not its blocks' means, not its shift state"""
    cfg = config(FULL)
    W = weights(cfg, seed=7, q_gain=3.0)
    a, b, c = tokens(70, cfg["vocab"], 4), tokens(45, cfg["vocab"], 5), tokens(50, cfg["vocab"], 6)
    wa, wb, wc = oracle(cfg, W, a), oracle(cfg, W, b), oracle(cfg, W, c)
    m = build(ctx, cfg, W, True, slots=2)
    sa, sb = m.acquire_slot(), m.acquire_slot()
    assert {sa, sb} == {0, 1}
    with pytest.raises(kf.KoifishError):
        m.acquire_slot()
    ga, gb, ia, ib = [], [], 0, 0
    for na, nb in [(30, 2), (1, 20), (2, 1), (37, 22)]:
        lg, _ = m.forward_rows(a[ia:ia + na], ia, slot=sa, rows=list(range(na)))
        ga.append(lg), (ia := ia + na)
        lg, _ = m.forward_rows(b[ib:ib + nb], ib, slot=sb, rows=list(range(nb)))
        gb.append(lg), (ib := ib + nb)
    assert rel(np.concatenate(ga), wa) < TOL[True] and rel(np.concatenate(gb), wb) < TOL[True]
    m.release_slot(sa)
    with pytest.raises(kf.KoifishError):
        m.release_slot(sa)
    sc = m.acquire_slot()
    assert sc == sa  # the slot that held the 70-token request: its rows, means and shift states are still in place
    assert rel(run_cut(m, c, [3, 2], slot=sc), wc) < TOL[True]
    m.close()


def test_batched_decode_of_unequal_requests(ctx):
    """three sequences of different lengths take one token each in one step -- some of them complete a block in it --: every row equals the
    sequence run alone"""
    cfg = config(FULL)
    W = weights(cfg, seed=8, q_gain=3.0)
    seqs = [tokens(n, cfg["vocab"], 10 + n) for n in (61, 17, 38)]
    want = [oracle(cfg, W, t) for t in seqs]
    m = build(ctx, cfg, W, True, slots=3)
    for s, t in enumerate(seqs):
        m.forward_rows(t[:-14], 0, slot=s)
    for k in range(14, 0, -1):
        lg, _ = m.forward_batch([t[len(t) - k] for t in seqs], [len(t) - k for t in seqs])
        for s, t in enumerate(seqs):
            assert rel(lg[s], want[s][len(t) - k]) < TOL[True], (s, k)
    m.close()


# ------------------------------------------------------------------------------------------------------------ shaped weights
@pytest.mark.parametrize("f32", [True, False])
def test_window_and_block_edges(ctx, f32, monkeypatch):
    """query norms x 6: the softmax is peaked, and a window or a block boundary one position off, mean rows that are left out or seen one
    position early or late move the logits far beyond the gate -- the oracle shows it first.  The framework then has to match in prompt panels
    (edges inside a panel and across panels), in small portions and in decoding, over several turns of the ring; the second layer's window
    is no multiple of its block, the third one's blocks are longer than its window."""
    cfg = config([layer(attn(heads=4, kv_heads=2, dim=16, vdim=16, window=23, pool=6), None), layer(attn(window=17, pool=7), moe()),
                  layer(attn(window=5, pool=19), None)])
    W = weights(cfg, seed=9, q_gain=6.0)
    toks = tokens(400, cfg["vocab"], 7)
    want = oracle(cfg, W, toks)
    gate = 3 * TOL[f32]
    for size, pool in ((24, 6), (22, 6), (23, 0), (23, 5), (23, 7)):
        assert rel(oracle(edited(cfg, lambda l: l["mixer"]["mask"].update(size=size, pool=pool)), W, toks), want) > gate, (size, pool)
    seen = ref.visible
    for late in (1, -1) if f32 else ():  # blocks seen one position late / early, in all three layers
        with monkeypatch.context() as mp:
            mp.setattr(ref, "visible", lambda i, S, P: (seen(i - late, S, P)[0], seen(i, S, P)[1]))
            assert rel(oracle(cfg, W, toks), want) > gate, (late, rel(oracle(cfg, W, toks), want))
    m = build(ctx, cfg, W, f32, max_seq=448)
    got = run_cut(m, toks, [64, 64, 23, 22, 24, 2, 2, 3, 64, 1, 6, 29])  # 304 in portions, then 96 decoded one by one
    assert close(got, want, f32)
    m.close()


@pytest.mark.parametrize("f32", [True, False])
def test_a_far_block_decides(ctx, f32):
    """a block of one repeated token A early in the sequence and, hundreds of positions later, a token B whose query is A's key (the keys read
    one half of the stream, the queries the other, through the same matrix): with query norms x 8 the block's mean key wins the softmax, so
    the late logits rest on a row made far back -- shown on the oracle by replacing the block -- in a prompt panel and in decoding, where the
    keys of a token are dealt to several CTAs"""
    cfg = config([layer(attn(heads=2, kv_heads=2, dim=32, vdim=32, window=40, pool=8), None)], width=64)
    W = weights(cfg, seed=18)
    K, V = W["l0.mix.k"][:, :32].clone(), cfg["vocab"]
    W["l0.mix.k"], W["l0.mix.q"] = torch.cat([K, 0 * K], 1), torch.cat([0 * K, K], 1)
    W["l0.mix.q.norm"], W["l0.mix.k.norm"] = torch.full((32,), 8.0), torch.ones(32)
    W["l0.shift"] = W["l0.shift"] * 0
    A, B = V - 2, V - 1
    W["embed"][B, 32:] = W["embed"][A, :32]
    toks = tokens(640, V - 2, 19)  # A and B do not occur by chance
    toks[48:56] = [A] * 8
    late = [300, 333, 470, 520, 600, 639]
    for t in late:
        toks[t] = B
    want = oracle(cfg, W, toks)
    gone = oracle(cfg, W, toks[:48] + toks[56:64] + toks[56:])
    assert min(rel(gone[[t]], want[[t]]) for t in late) > 3 * TOL[f32]
    m = build(ctx, cfg, W, f32, max_seq=700)
    assert close(run_cut(m, toks, [64] * 8 + [3, 2]), want, f32)  # 517 in portions, then 123 decoded one by one
    m.close()


@pytest.mark.parametrize("hd, heads, kv", [(64, 4, 2), (128, 2, 1), (64, 3, 3)])
def test_panel_attention_on_tensor_cores(ctx, hd, heads, kv):
    """bf16, head size 64 / 128: panels of 16 tokens and more run the tile kernel (a peaked softmax, gates that matter, window and block edges
    that fall inside 64-row tiles and inside panels, more blocks than one tile of keys, panels that start inside a tile, a ring that turns
    several times); smaller portions and decoded tokens run the general kernel on the same rows"""
    cfg = config([layer(attn(heads=heads, kv_heads=kv, dim=hd, vdim=hd, window=75, pool=3), None)], width=64, vocab=80)
    W = weights(cfg, seed=16, q_gain=4.0)
    toks = tokens(400, cfg["vocab"], 17)
    want = oracle(cfg, W, toks)
    for size, pool in ((74, 3), (75, 0), (75, 4)):
        assert rel(oracle(edited(cfg, lambda l: l["mixer"]["mask"].update(size=size, pool=pool)), W, toks), want) > 2 * TOL[False]
    assert rel(oracle(cfg, dict(W, **{"l0.mix.g": W["l0.mix.g"] * 0}), toks), want) > 2 * TOL[False]
    m = build(ctx, cfg, W, False, max_seq=420)
    assert close(run_cut(m, toks, [64, 17, 3, 64, 30, 2, 16, 40, 64, 64]), want, False)
    m.close()


def test_long_decoding_through_the_ring(ctx):
    """three tokens of prompt, then 300 decoded one by one with windows and blocks far below the length (ring of 13 + 64 - 1 rows: four turns,
    75 blocks), all positions checked"""
    cfg = config([layer(attn(window=13, pool=4), moe()), layer(attn(window=13, pool=4), moe(), weights_of=0), layer(attn(window=64, pool=9), None)])
    W = weights(cfg, seed=10, q_gain=3.0)
    toks = tokens(303, cfg["vocab"], 8)
    m = build(ctx, cfg, W, True, max_seq=320)
    assert m.info.kv_bytes < 2 * 4 * (2 * ((76 + 80) * 44 + 48) + (127 + 35) * 44 + 48 + 64)  # rings and mean rows, not max_seq rows
    assert rel(run_cut(m, toks, [3]), oracle(cfg, W, toks)) < TOL[True]
    m.close()


def test_context_that_fills_the_model(ctx):
    """max_seq below window + panel: the ring is cut to max_seq rows; decoded to the last position, blocks still count"""
    cfg = config([layer(attn(window=50, pool=7), moe()), layer(attn(window=95, pool=1), None), layer(attn(window=96, pool=2), None)])
    W = weights(cfg, seed=12, q_gain=3.0)
    toks = tokens(96, cfg["vocab"], 8)
    m = build(ctx, cfg, W, True, max_seq=96)
    assert rel(run_cut(m, toks, [64, 9]), oracle(cfg, W, toks)) < TOL[True]
    m.close()


# ------------------------------------------------------------------------------------------------------------ kernels on their own
class Route(C.Structure):
    _fields_ = [("table", C.c_void_p), ("idx", C.c_void_p), ("offsets", C.c_void_p), ("entry_slot", C.c_void_p), ("slot_row", C.c_void_p), ("slot_group", C.c_void_p),
                ("work", C.c_void_p), ("wgt", C.c_void_p), ("experts", C.c_int), ("top", C.c_int)]


@pytest.mark.parametrize("M", [1, 5, 64, 300])
def test_dispatch_tables_of_several_layers(ctx, M):
    """kf_moe_route_table: three layers of different sizes in one call, the one-block form and the many-token form"""
    rs = np.random.RandomState(M)
    V, sizes = 50, [(12, 3), (1, 1), (70, 6)]
    toks = rs.randint(0, V, M).astype(np.int32)
    keep, routes, tabs = [], (Route * 3)(), []
    for r, (E, top) in enumerate(sizes):
        tab = np.stack([rs.permutation(E)[:top] for _ in range(V)]).astype(np.int32)
        n = M * top
        b = [ctx.array(tab)] + [ctx.zeros(k * 4) for k in (n, E + 1, n, n, n, n + E, n)]
        keep.append(b), tabs.append(tab)
        routes[r] = Route(*[x.ptr for x in b], E, top)
    td, rd = ctx.array(toks), ctx.array(np.frombuffer(bytes(routes), dtype=np.uint8))
    ctx.check(ctx.lib.kf_moe_route_table(ctx.h, rd.ptr, 3, 70, 6, td.ptr, M), "kf_moe_route_table")
    for r, (E, top) in enumerate(sizes):
        n = M * top
        idx, off, entry, row, grp = (keep[r][k].numpy(np.int32, (s,)) for k, s in ((1, n), (2, E + 1), (3, n), (4, n), (5, n)))
        want = tabs[r][toks].reshape(-1)
        assert np.array_equal(idx, want) and np.allclose(keep[r][7].numpy(np.float32, (n,)), 1.0 / top)
        assert off[0] == 0 and off[E] == n and np.array_equal(np.diff(off), np.bincount(want, minlength=E))
        assert np.array_equal(np.sort(entry), np.arange(n)) and np.array_equal(grp[entry], want) and np.array_equal(row[entry], np.arange(n) // top)
        assert np.all(np.diff(grp) >= 0)


def test_token_shift_kernel_over_several_sequences(ctx):
    rs = np.random.RandomState(2)
    nseq, T, dim = 3, 9, 37
    h = rs.randn(nseq * T, dim).astype(np.float32)
    w = bf16_grid(torch.from_numpy(rs.randn(dim).astype(np.float32)))
    tail = rs.randn(4, dim + 3).astype(np.float32)
    pos = np.concatenate([np.arange(T), np.arange(T) + 5, np.concatenate([np.arange(4) + 2, np.arange(5)])]).astype(np.int32)  # the third one restarts inside
    slot = np.repeat(np.array([2, 0, 3]), T).astype(np.int32)
    hd, wd, td, pd, sd, out = ctx.array(h), ctx.array(bits(w)), ctx.array(tail), ctx.array(pos), ctx.array(slot), ctx.empty(nseq * T * dim * 4)
    ctx.check(ctx.lib.kf_token_shift(ctx.h, out.ptr, 1, hd.ptr, dim, wd.ptr, td.ptr, dim + 3, pd.ptr, sd.ptr, nseq, T, dim), "kf_token_shift")
    got, new = out.numpy(np.float32, (nseq * T, dim)), td.numpy(np.float32, (4, dim + 3))
    for s in range(nseq):
        prev = tail[slot[s * T], :dim]
        for t in range(T):
            m = s * T + t
            if pos[m] == 0:
                prev = np.zeros(dim, dtype=np.float32)
            assert np.abs(got[m] - (h[m] + (prev - h[m]) * w.numpy())).max() < 1e-5
            prev = h[m]
        assert np.array_equal(new[slot[s * T], :dim], h[s * T + T - 1])
    assert np.array_equal(new[1], tail[1]) and np.array_equal(new[:, dim:], tail[:, dim:])


def test_postnorm_step_options(ctx):
    """kf_postnorm_residual_ex with two branches, a weight per entry stored around zero, a factor and the shift; kf_experts_postnorm_residual
    without a shared expert -- what the stack does not use"""
    rs = np.random.RandomState(3)
    M, dim, top = 5, 90, 3
    x, a, b = (rs.randn(M, dim).astype(np.float32) for _ in range(3))
    w, sh = (bf16_grid(torch.from_numpy(rs.randn(dim).astype(np.float32))) for _ in range(2))
    tail = rs.randn(6, dim).astype(np.float32)
    pos, slot = np.array([4, 0, 9, 1, 7], dtype=np.int32), np.array([5, 0, 3, 1, 4], dtype=np.int32)
    norm = lambda v: v / np.sqrt((v * v).mean(-1, keepdims=True) + 1e-3)
    xd, ad, bd, wd, shd, td, pd, sd, act = ctx.array(x), ctx.array(a), ctx.array(b), ctx.array(bits(w)), ctx.array(bits(sh)), ctx.array(tail), ctx.array(pos), ctx.array(slot), ctx.empty(M * dim * 4)
    ctx.check(ctx.lib.kf_postnorm_residual_ex(ctx.h, xd.ptr, act.ptr, 1, ad.ptr, dim, 0.7, bd.ptr, dim, -1.3, wd.ptr, 1.0, 0, 0.45, M, dim, 1e-3, shd.ptr, td.ptr, dim, pd.ptr, sd.ptr),
              "kf_postnorm_residual_ex")
    want = x + 0.45 * norm(0.7 * a - 1.3 * b) * (1.0 + w.numpy())
    assert np.abs(xd.numpy(np.float32, (M, dim)) - want).max() < 1e-5
    prev = np.where((pos == 0)[:, None], 0.0, tail[slot])
    assert np.abs(act.numpy(np.float32, (M, dim)) - (want + (prev - want) * sh.numpy())).max() < 2e-5
    assert np.abs(td.numpy(np.float32, (6, dim))[slot] - want).max() < 1e-5
    y = rs.randn(M * top, dim).astype(np.float32)
    entry, wgt = rs.permutation(M * top).astype(np.int32), rs.rand(M * top).astype(np.float32)
    xd, yd, ed, gd, act = ctx.array(x), ctx.array(y), ctx.array(entry), ctx.array(wgt), ctx.empty(M * dim * 2)
    ctx.check(ctx.lib.kf_experts_postnorm_residual(ctx.h, xd.ptr, act.ptr, 0, yd.ptr, ed.ptr, gd.ptr, None, top, wd.ptr, 0.0, 1, 2.0, M, dim, 1e-3, None, None, 0, None, None),
              "kf_experts_postnorm_residual")
    s = (y[entry] * wgt[:, None]).reshape(M, top, dim).sum(1)
    want = x + 2.0 * norm(s) * w.numpy()[0]
    assert np.abs(xd.numpy(np.float32, (M, dim)) - want).max() < 2e-5
    assert np.abs((act.numpy(np.uint16, (M, dim)).astype(np.uint32) << 16).view(np.float32) - want).max() < 2e-2


@pytest.mark.parametrize("layout", [0, 1])
def test_heads_prepare_and_window_with_everything(ctx, layout):
    """kf_qk_heads_prepare with a rotation + kf_attn_window_ex with cap, sink, factor, blocks and gate together (what the stack does not combine),
    a float ring, several slots, one step per call and all in one call: both give the same rows"""
    rs = np.random.RandomState(5)
    T, H, G, dk, dv, rot, win, pool, ring = 23, 4, 2, 12, 6, 8, 7, 3, 32
    W = G * (dk + dv)
    nq, nk, nv = H * dk, G * dk, G * dv
    x = rs.randn(T, nq + nk + nv).astype(np.float32)
    qw, kw = (bf16_grid(torch.from_numpy(1 + rs.randn(dk).astype(np.float32) * 0.3)) for _ in range(2))
    freq = (50.0 ** (-2.0 * np.arange(rot // 2) / rot)).astype(np.float64)
    stride = (ring + 10) * W
    gate, sink = rs.randn(T, H + 3).astype(np.float32), bf16_grid(torch.from_numpy(rs.randn(H).astype(np.float32)))
    qwd, kwd, fd, gd, skd = ctx.array(bits(qw)), ctx.array(bits(kw)), ctx.array(freq), ctx.array(gate), ctx.array(bits(sink))

    def step(cache, lo, hi, slot, one):
        xd = ctx.array(x[lo:hi])
        pd, sd = ctx.array(np.arange(lo, hi, dtype=np.int32)), ctx.array(np.full(hi - lo, slot, dtype=np.int32))
        ctx.check(ctx.lib.kf_qk_heads_prepare(ctx.h, xd.ptr, nq + nk + nv, H, G, dk, dv, qwd.ptr, kwd.ptr, 1e-5, rot, fd.ptr, 1.5, layout, cache.ptr, 1, stride, ring, pool,
                                              one, None, pd.ptr, sd.ptr, hi - lo), "kf_qk_heads_prepare")
        out = ctx.empty((hi - lo) * H * dv * 4)
        gl = ctx.array(gate[lo:hi])
        ctx.check(ctx.lib.kf_attn_window_ex(ctx.h, out.ptr, 1, H * dv, xd.ptr, nq + nk + nv, cache.ptr, 1, stride, ring, skd.ptr, pd.ptr, sd.ptr, hi - lo, H, G, dk, dv, 0.4, 2.0,
                                            win, 64, 0.5, pool, gl.ptr, H + 3), "kf_attn_window_ex")
        return out.numpy(np.float32, (hi - lo, H, dv))

    whole, single = ctx.zeros(2 * stride * 4), ctx.zeros(2 * stride * 4)
    a = step(whole, 0, T, 1, 0)
    b = np.concatenate([step(single, t, t + 1, 0, 1) for t in range(T)])
    ra, rb = whole.numpy(np.float32, (2, stride))[1], single.numpy(np.float32, (2, stride))[0]
    assert np.array_equal(ra, rb) and np.abs(a - b).max() < 1e-5

    def finish(v, w, p):
        v = v / np.sqrt((v * v).mean(-1, keepdims=True) + 1e-5) * w.numpy()
        out, ang = v.copy(), p * freq
        ia = np.arange(0, rot, 2) if layout == 0 else np.arange(rot // 2)
        ib = ia + 1 if layout == 0 else ia + rot // 2
        out[:, ia] = 1.5 * (v[:, ia] * np.cos(ang) - v[:, ib] * np.sin(ang))
        out[:, ib] = 1.5 * (v[:, ib] * np.cos(ang) + v[:, ia] * np.sin(ang))
        return out

    xx = x.astype(np.float64)
    q = np.stack([finish(xx[t, :nq].reshape(H, dk), qw, t) for t in range(T)])
    k = np.stack([finish(xx[t, nq:nq + nk].reshape(G, dk), kw, t) for t in range(T)])
    v = xx[:, nq + nk:].reshape(T, G, dv)
    for t in range(T):
        blocks, toks = ref.visible(t, win, pool)
        keys = np.stack([k[c * pool:(c + 1) * pool].mean(0) for c in blocks] + [k[j] for j in toks])
        vals = np.stack([v[c * pool:(c + 1) * pool].mean(0) for c in blocks] + [v[j] for j in toks])
        for h in range(H):
            g = h // (H // G)
            s = np.exp(2.0 * np.tanh(keys[:, g] @ q[t, h] * 0.4 / 2.0))
            want = 0.5 / (1 + np.exp(-gate[t, h])) * (s[:, None] * vals[:, g]).sum(0) / (s.sum() + np.exp(sink.numpy()[h]))
            assert np.abs(a[t, h] - want).max() < 2e-5, (t, h)


@pytest.mark.parametrize("window, pool, cap, sink", [(40, 4, 0.0, False), (40, 4, 3.0, True), (0, 0, 0.0, True), (100, 0, 0.0, False)])
def test_panel_kernel_against_the_general_one(ctx, window, pool, cap, sink):
    """kf_attn_pooled_prefill and kf_attn_window_ex on the same bf16 rows, with and without blocks, window, cap and sink"""
    rs = np.random.RandomState(8)
    T, p0, H, G, hd, ring = 150, 77, 4, 2, 64, 256
    W = 2 * G * hd
    stride = (ring + 64) * W
    f32 = lambda u: (u.astype(np.uint32) << 16).view(np.float32)
    rows = bits(torch.from_numpy(rs.randn(stride).astype(np.float32)))
    q = f32(bits(torch.from_numpy(3 * rs.randn(T, H * hd).astype(np.float32))))
    gate = rs.randn(T, H).astype(np.float32)
    snk = ctx.array(bits(torch.from_numpy(np.float32([0.5, 2.0, -1.0, 3.0])))) if sink else None
    cd, qd, qbd, gd = ctx.array(rows), ctx.array(q), ctx.array(bits(torch.from_numpy(q))), ctx.array(gate)
    pd, sd = ctx.array(np.arange(p0, p0 + T, dtype=np.int32)), ctx.array(np.zeros(T, dtype=np.int32))
    o1, o2 = ctx.empty(T * H * hd * 4), ctx.empty(T * H * hd * 2)
    sp = snk.ptr if sink else None
    ctx.check(ctx.lib.kf_attn_window_ex(ctx.h, o1.ptr, 1, H * hd, qd.ptr, H * hd, cd.ptr, 0, stride, ring, sp, pd.ptr, sd.ptr, T, H, G, hd, hd, 0.125, cap, window, p0 + T, 1.0, pool,
                                        gd.ptr, H), "kf_attn_window_ex")
    ctx.check(ctx.lib.kf_attn_pooled_prefill(ctx.h, o2.ptr, H * hd, qbd.ptr, cd.ptr, stride, ring, sp, pd.ptr, sd.ptr, T, H, G, hd, 0.125, cap, window, pool, gd.ptr, H, 1.0),
              "kf_attn_pooled_prefill")
    a, b = o1.numpy(np.float32, (T, H * hd)), f32(o2.numpy(np.uint16, (T, H * hd)))
    assert np.abs(a - b).max() < 1e-2 * np.abs(a).max()


# ------------------------------------------------------------------------------------------------------------ entry points
def test_greedy_generation(ctx):
    cfg = config(FULL)
    W = weights(cfg, seed=11)
    prompt = tokens(70, cfg["vocab"], 9)  # longer than a panel
    seq = list(prompt)
    for _ in range(12):
        seq.append(int(np.argmax(oracle(cfg, W, seq)[-1])))
    m = build(ctx, cfg, W, True)
    out, why = m.generate(prompt, 12)
    assert out == seq[len(prompt):] and why == 2
    # the device-resident loop from the same prompt
    m.forward(prompt[:64], np.arange(64), seq_mode=2, want_logits=False)
    m.forward(prompt[64:], np.arange(64, 70), seq_mode=2, want_logits=False, want_next=True)
    m.decode_loop(11, 1)
    ctx.sync()
    t, p = m.read_state(1)
    assert int(t[0]) == seq[-1] and int(p[0]) == len(seq) - 1
    m.close()


def test_tables_of_ids_are_checked_saved_and_loaded(ctx, tmp_path):
    cfg = config([layer(attn(), moe()), layer(attn(), moe(), weights_of=0)], width=32)
    W = weights(cfg, seed=13)
    toks = tokens(20, cfg["vocab"], 3)
    m = build(ctx, cfg, W, False)
    want = run_cut(m, toks, [20])
    bad = W["l0.mlp.table"].numpy().copy()
    bad[7, 1] = 6
    with pytest.raises(kf.KoifishError, match="every id"):
        m.set_tensor("l0.mlp.table", bad)
    bad[7, 1] = -1
    with pytest.raises(kf.KoifishError, match="every id"):
        m.set_tensor("l0.mlp.table", bad)
    with pytest.raises(kf.KoifishError, match="table of 32-bit ids"):
        m.set_tensor("l0.mlp.table", np.zeros((96, 2), dtype=np.uint16))
    with pytest.raises(kf.KoifishError, match="cannot be a weight"):
        m.set_tensor("l0.shift", np.zeros((1, 32), dtype=np.int32))
    with pytest.raises(kf.KoifishError, match="expected a table"):
        m.set_tensor("l0.mlp.table", np.zeros((2, 96), dtype=np.int32))
    assert np.array_equal(run_cut(m, toks, [20]), want)
    m.save(str(tmp_path / "w.blob"))
    m.save_kun(str(tmp_path / "w.kun"))
    for load in ("load", "load_kun"):
        n = kf.Model(ctx, {"hf_config": cfg, "gpt": {"max_seq_len": 256, "max_batch": 2, "max_prefill": 64, "logit_rows": 64}})
        getattr(n, load)(str(tmp_path / ("w.blob" if load == "load" else "w.kun")))
        assert np.array_equal(run_cut(n, toks, [20]), want)
        n.close()
    m.init_random()  # synthetic tables name experts that exist, each once per row
    assert np.isfinite(run_cut(m, toks, [20])).all()
    m.close()
    ent = st_entries(W)
    k = [e[0] for e in ent].index("l0.mlp.table")
    for a, words in (((ent[k][0], "I32", bad), "every id"), ((ent[k][0], "F32", ent[k][2].astype(np.float32)), "stored as I32")):
        d = tmp_path / ("bad_" + a[1])
        d.mkdir()
        (d / "config.json").write_text(json.dumps(cfg))
        write_safetensors(str(d / "model.safetensors"), ent[:k] + [a] + ent[k + 1:])
        with pytest.raises(kf.KoifishError, match=words):
            kf.from_pretrained(ctx, str(d), max_seq_len=64)


def test_command_line_on_a_checkpoint_folder(ctx, tmp_path):
    """config.json + model.safetensors on disk -> `generate` and `trace` of the command line, both number formats; optional keys left out of
    the file (kv_heads, vdim, scale, shared expert, residual factor) take their defaults"""
    cfg = config([layer(attn(heads=3, kv_heads=3, dim=8, vdim=8), moe(shared=0)), layer(attn(), None), layer(attn(), None, weights_of=1)], mult=1.0)
    W = weights(cfg, seed=12)
    disk = json.loads(json.dumps(cfg))
    disk.pop("residual_mult")
    a0 = disk["layers"][0]["mixer"]
    a0.pop("kv_heads"), a0.pop("vdim"), a0.pop("scale")
    d = tmp_path / "ckpt"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(disk))
    write_safetensors(str(d / "model.safetensors"), st_entries(W))
    a, b = tokens(75, cfg["vocab"], 13), tokens(9, cfg["vocab"], 14)
    wa, wb = oracle(cfg, W, a), oracle(cfg, W, b)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:70], "want": [0, 5, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[70:72], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[72:], "want": [2, 1]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b, "want": [8]}], "end": ["y"]}]
    env = dict(os.environ, PYTHONPATH=ROOT)
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / ("out_" + dtype)
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(d), "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=env, timeout=900)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        assert not (out / "1.f32").exists()
        f = lambda n: np.fromfile(str(out / ("%d.f32" % n)), dtype="<f4").reshape(-1, cfg["vocab"])
        got, want = np.concatenate([f(0), f(2), f(3)]), np.concatenate([wa[[0, 5, 69]], wa[[74, 73]], wb[[8]]])
        assert close(got, want, dtype == "float32")
    r = subprocess.run([sys.executable, "-m", "koifish_b200.cli", "generate", "--model", str(d), "--ids", ",".join(map(str, b)), "--max-new-tokens", "5"],
                       capture_output=True, text=True, env=env, cwd=ROOT, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    seq = list(b)
    for _ in range(5):
        seq.append(int(np.argmax(oracle(cfg, W, seq)[-1])))
    got = json.loads(r.stdout.strip().splitlines()[-1])["tokens"]
    assert len(got) == 5 and got[0] == seq[len(b)]  # bf16 serving: the first token is far from a tie; later ones may legitimately differ

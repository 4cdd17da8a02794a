"""The Pipesun design in the engine against the plain implementation (tests/plain/pipesun_plain.py): every mechanism alone,
then whole models under every way of cutting the work.  Needs a B200; float32 (true 32-bit) and bfloat16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from helpers import TOL, random_tokens, rel_l2, rows_close, write_folder
from pipesun_cases import as_numpy, attention, latent, layer, make_config, model, random_weights
from plain import pipesun_plain as P
from test_desalorn_gpu import BOTH, DT, WIDTH, bind, drive, inputs, make_ctx, plain_weights, run_in_pieces, t64, weights_for

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
EPS = 1e-5


# --------------------------------------------------------------------------- #
# mechanisms alone
# --------------------------------------------------------------------------- #
@pytest.mark.parametrize("W,rows_per_block", [(48, 0), (51, 0), (64, 3), (256, 4), (1000, 2), (2048, 4), (4096, 1), (5000, 0), (7, 5)])
def test_norm_and_token_shift(W, rows_per_block):
    """Three unequal sequences in slots out of order: whole, in portions down to one token, in batches where one joins late; the
    state holds the last row's normed values before the shift, the other slots' states stay as they were; then a slot used again."""
    from titan_b200 import kernels as K
    from titan_b200.engine.batch import StepEntry
    g = torch.Generator().manual_seed(W)
    w, mu = torch.randn(W, generator=g) * 0.3 + 1, torch.randn(W, generator=g)
    lens, slots = [37, 5, 12], [4, 0, 2]
    xs = [torch.randn(n, W, generator=g) * 3 for n in lens]
    normed = [P.rms_norm(x.double().numpy(), w.double().numpy(), EPS) for x in xs]
    want = [t64(P.token_shift(n, mu.double().numpy())) for n in normed]
    for dtype in BOTH:
        state = torch.full((6, W), 7.0, device="cuda")
        for plan in ([lens], [[20, 0, 5], [1, 2, 2], [16, 3, 0], [0, 0, 5]], [[1, 1, 1]] * 37):
            state[slots] = 0.0
            at, got = [0, 0, 0], [[], [], []]
            for sizes in plan:
                take = [(i, min(n, lens[i] - at[i])) for i, n in enumerate(sizes) if n and at[i] < lens[i]]
                ctx = make_ctx([StepEntry(slots[i], [0] * n, []) for i, n in take], [at[i] for i, _ in take], DT[dtype])
                x = torch.cat([xs[i][at[i]:at[i] + n] for i, n in take]).cuda()
                h = torch.empty(x.shape, dtype=DT[dtype], device="cuda")
                K.shift_norm(x, w.cuda(), EPS, mu.cuda(), h, state, ctx.layout, ctx.stream, rows_per_block)
                o = 0
                for i, n in take:
                    got[i].append(h[o:o + n].float().cpu())
                    o, at[i] = o + n, at[i] + n
                    rows_close(state[slots[i]][None], t64(normed[i][at[i] - 1:at[i]]), "float32", "state")
            for i in range(3):
                rows_close(torch.cat(got[i]), want[i], dtype, f"sequence {i}", row_factor=6.0)
            assert bool((state[[1, 3, 5]] == 7.0).all()), "a slot that is not in the batch was written"


@pytest.mark.parametrize("W,T", [(48, 3), (51, 9), (256, 1), (1000, 40), (2048, 300), (4096, 2), (4096, 400), (8192, 5), (12000, 400), (20000, 2)])
def test_a_sublayers_output_joins_the_residual_stream(W, T):
    """x += rms(y) w with y left zeroed, alone; with the next sublayer's normed rows; with the average over depth of one, two and
    five earlier rows (the first kept in the same launch or before); with the shifted rows of the next block's mixer and its states."""
    from titan_b200 import kernels as K
    g = torch.Generator().manual_seed(W + T)
    n = lambda *s: torch.randn(*s, generator=g)
    y, x, wb, w2, mu = n(T, W) * 5, n(T, W), n(W), n(W), n(W)
    d = lambda t: t.double().numpy()
    joined = d(x) + P.rms_norm(d(y), d(wb), EPS)
    slots = torch.randperm(T + 3, generator=g)[:T].to(torch.int32)
    states = n(T + 3, W)
    for dtype in BOTH:
        def run(**kw):
            xd, yd = x.cuda().clone(), y.cuda().clone()
            K.sandwich_join(yd, wb.cuda(), EPS, xd, K.current_stream(), **kw)
            assert float(yd.abs().max()) == 0.0
            return xd
        rows_close(run(), t64(joined), "float32", "the sum alone")
        h, keep = torch.empty(T, W, dtype=DT[dtype], device="cuda"), torch.empty(T, W, device="cuda")
        rows_close(run(pre_w=w2.cuda(), pre_eps=1e-3, h=h, keep=keep), t64(joined), "float32", "with a norm behind it")
        assert torch.equal(keep.cpu(), x)
        rows_close(h, t64(P.rms_norm(joined, d(w2), 1e-3)), dtype, "normed rows")
        for depth in (1, 2, 5):
            hist, dw = n(depth + 1, T, W), n(depth + 1)
            for first_now in (False, True):
                H = hist.cuda().clone()
                rows = [d(hist[j]) for j in range(depth)] + [joined]
                if first_now:
                    rows[0] = d(x)
                mean = P.depth_average(rows, d(dw))
                st = states.cuda().clone()
                xd = run(history=H, depth=depth, depth_w=dw.cuda(), keep=H[0] if first_now else None, pre_w=w2.cuda(), pre_eps=EPS, h=h, mu=mu.cuda(), state=st,
                         slot_of_row=slots.cuda())
                rows_close(xd, t64(mean), "float32", f"average over {depth + 1}")
                rows_close(H[depth], t64(joined), "float32", "the new row of the history")
                assert torch.equal(H[0].cpu(), x if first_now else hist[0])
                normed = P.rms_norm(mean, d(w2), EPS)
                before = d(states)[slots.numpy()]
                rows_close(h, t64(normed + (before - normed) * d(mu)), dtype, "shifted rows", row_factor=8.0)
                rows_close(st[slots.long().cuda()], t64(normed), "float32", "states")
                rest = torch.ones(T + 3, dtype=torch.bool)
                rest[slots.long()] = False
                assert torch.equal(st.cpu()[rest], states[rest])
            short = hist[:depth].cuda().clone()                       # the last layer: nobody reads its row again, the history has no place for it
            rows_close(run(history=short, depth=depth, depth_w=dw.cuda()), t64(P.depth_average([d(hist[j]) for j in range(depth)] + [joined], d(dw))), "float32", "last layer")


def diff_spec(H, G, dim, vdim, scale, diff, reader=False, eps=EPS):
    from titan_b200.config import MixerSpec, NormSpec, PositionSpec
    return MixerSpec("differential_attention", WIDTH, H, G, dim, qk_norm=NormSpec("rmsnorm", dim, eps, "{}.norm"), softmax_scale=scale, prefix="d.",
                     position=PositionSpec("none"), cache_from=0 if reader else None,
                     names=tuple((r, r) for r in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2")),
                     extra=(("value_dim", vdim), ("diff", diff), ("out_eps", eps), ("bias", True)))


def diff_weights(mixer, seed, dim):
    w = weights_for(mixer, seed)
    g = torch.Generator().manual_seed(seed + 1)
    for r in ("lq1", "lk1", "lq2", "lk2"):
        w["d." + r] = (torch.randn(dim, generator=g) * 0.6 / dim ** 0.25).to(torch.bfloat16).float()
    return w


DIFF_SIZES = [
    (4, 2, 12, 20, 0.2),                    # rows of 32, keys and values padded
    (3, 3, 7, 5, 0.0),                      # as many kv heads as heads, no multiples of anything
    (2, 1, 3, 29, 0.8),                     # values far wider than both maps
    (1, 1, 16, 32, 0.5),
    (6, 2, 64, 128, 0.3),                   # rows of 128: tensor cores in bfloat16, six maps on a kv head
    (8, 1, 60, 120, 0.5),                   # padded to 128, sixteen maps on one kv head
    (9, 1, 64, 100, 0.3),                   # eighteen maps on a kv head: more than the tensor-core decode kernel takes
    (2, 2, 32, 64, 0.45),                   # rows of 64
    (2, 1, 25, 40, 0.1),                    # padded to 64
    (2, 1, 100, 200, 0.4),                  # rows of 208
    (1, 1, 150, 260, 0.4),                  # rows of 304: the wide instantiation
]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,dim,vdim,diff", DIFF_SIZES)
def test_differential_attention_with_a_reader_of_its_keys(dtype, H, G, dim, vdim, diff):
    """Biases, norms a map, both maps, lambda, the unit norm and the factor; and a second mixer with its own queries, lambda, scale
    and factor on the first one's keys and values: whole prompts of two unequal sequences, portions down to two tokens, single
    tokens across a page's border; then the slots again (freed pages overwritten)."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    own, reader = MIXERS.build(diff_spec(H, G, dim, vdim, 0.4, diff)), MIXERS.build(diff_spec(H, G, dim, vdim, 0.25, 0.15, reader=True))
    wo, wr = diff_weights(own, 3, dim), diff_weights(reader, 13, dim)
    bind(own, wo, DT[dtype]), bind(reader, wr, DT[dtype])
    mo, mr = attention(H, G, dim, vdim, 0.4, diff), attention(H, G, dim, vdim, 0.25, 0.15)
    lens = [150, 71]
    xs = inputs(lens, 5)
    Wo, Wr = plain_weights(wo, "d."), plain_weights(wr, "d.")
    want = []
    for x in xs:
        kv = P.keys_and_values(x.numpy(), Wo, "", mo, EPS)
        want.append(torch.cat([t64(P.differential_attention(x.numpy(), Wo, "", mo, EPS)), t64(P.differential_attention(x.numpy(), Wr, "", mr, EPS, kv))], dim=1))
    cache = SequenceCache([own.cache_need()], 1024, 4, 512, DT[dtype], "cuda", mark_freed=True)
    assert reader.cache_need() is None

    def step(h, ctx):
        a, b = torch.zeros(h.shape[0], WIDTH, device="cuda"), torch.zeros(h.shape[0], WIDTH, device="cuda")
        own.forward(h, ctx, cache.view_for_layer(0), a)
        reader.forward(h, ctx, cache.view_for_layer(0), b)
        return torch.cat([a, b], dim=1)
    for sizes in ([lens], [[60, 33], [50, 2], [2, 2], [2, 30]], [[1, 1]]):
        got = drive(step, cache, xs, dtype, sizes)
        for i in range(2):
            rows_close(got[i], want[i], dtype, f"sequence {i}, portions {sizes}", row_factor=6.0)


def mixer_step(mixer, cache):
    def step(h, ctx):
        out = torch.zeros(h.shape[0], WIDTH, device="cuda")
        mixer.forward(h, ctx, cache.view_for_layer(0), out)
        return out
    return step


LAST = 229
FAR = [0, 1, 63, 64, 65, 127, 128, 191, 192, LAST - 1]


def through_every_cut(step, cache, x, far, dtype, want):
    n = x.shape[0]
    for sizes, what in (([[n]], "in a prompt"), ([[n - 1]], "decoded alone"), ([[far + 1], [max(1, n - far - 3)], [2]], "in portions"), ([[max(1, far)]], "decoded from the key on")):
        rows_close(drive(step, cache, [x], dtype, sizes)[0][-1:], want[-1:], dtype, what, row_factor=6.0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("dim", [16, 32, 64])
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("far", FAR)
def test_one_far_key_decides_one_map(dtype, dim, which, far):
    """One map's key matrix is minus its query matrix and the last token's input row is minus that of position ``far``: that key,
    among hundreds, takes nearly all of that map's weight, while the other map's queries are zero (a mean over all values).  The
    last output is then that key's value against the mean, with the sign and the factor of its map; a key lost at a page's border
    or at the sequence's start, or a map taken for the other, gives another row.  In a prompt, decoded, in portions."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    H, vdim = 2, 2 * dim
    mixer = MIXERS.build(diff_spec(H, 1, dim, vdim, 40.0 / dim, 0.5))
    w = diff_weights(mixer, 7, dim)
    q = w["d.q"].reshape(H, 2, dim, WIDTH)
    q[:, 1 - which] = 0.0
    q[1] = q[0]                                                    # both heads ask alike: one key head serves them
    w["d.q"] = q.reshape(2 * H * dim, WIDTH).contiguous()
    k = w["d.k"].reshape(2, dim, WIDTH)
    k[which] = -q[0, which]
    w["d.k"] = k.reshape(2 * dim, WIDTH).contiguous()
    for r in ("q", "k", "v"):
        w[f"d.{r}.b"] = w[f"d.{r}.b"] * 0.0
    w["d.q.norm"], w["d.k.norm"] = torch.ones(dim), torch.ones(dim)
    bind(mixer, w, DT[dtype])
    m = attention(H, 1, dim, vdim, 40.0 / dim, 0.5)
    x = inputs([LAST + 1], 8)[0]
    x[-1] = -x[far]
    W = plain_weights(w, "d.")
    want = t64(P.differential_attention(x.numpy(), W, "", m, EPS))
    v = x.numpy() @ W["v"].T
    maps = [v[far], v.mean(axis=0)] if which == 0 else [v.mean(axis=0), v[far]]
    alone = P.map_difference(maps[0], maps[1], P.lambda_of(W, "", 0.5), 0.5, EPS)
    assert rel_l2(t64(np.tile(alone, H) @ W["o"].T), want[-1]) < 0.2, "the test's weights do not single the key out"
    cache = SequenceCache([mixer.cache_need()], 1024, 4, 512, DT[dtype], "cuda", mark_freed=True)
    through_every_cut(mixer_step(mixer, cache), cache, x, far, dtype, want)


@pytest.mark.parametrize("source", ["step", "cache"])
@pytest.mark.parametrize("hd,kernel", [(128, "tc"), (128, "mma"), (64, "mma")])
def test_tensor_core_prompts_keep_sixteen_bits_of_a_weight(hd, kernel, source):
    """Grouped-query attention in bfloat16 with float32 rows out, against float64 on the same rounded queries, keys and values: with
    the weights in two halves the error is a hundredth of what one bfloat16 rounding of the weights costs."""
    from titan_b200 import kernels as K
    from titan_b200.cache import SequenceCache
    from titan_b200.cache.groups import CacheNeed
    from titan_b200.engine.batch import StepEntry
    nh, nkv, n = 4, 2, 333
    g = torch.Generator().manual_seed(hd)
    rows = torch.randn(n, (nh + 2 * nkv) * hd, generator=g).to(torch.bfloat16)
    cache = SequenceCache([CacheNeed("kv", nkv, hd)], 1024, 2, 512, torch.bfloat16, "cuda")
    slot = cache.alloc_slot()
    cache.reserve({slot: n})
    ctx = make_ctx([StepEntry(slot, [0] * n, [])], [0], torch.bfloat16)
    group, index = cache.view_for_layer(0)
    view = K.KvView(group.layer_storage(index).data_ptr(), group.table.data_ptr(), group.table_width, 0, group.page_size, group.num_pages, nkv, hd)
    d = rows.cuda()
    K.kv_append(d[:, nh * hd:], view, ctx.layout.c_struct(), ctx.stream)
    r = rows.double()
    q, k, v = r[:, :nh * hd].reshape(n, nh, hd), r[:, nh * hd:(nh + nkv) * hd].reshape(n, nkv, hd), r[:, (nh + nkv) * hd:].reshape(n, nkv, hd)
    want = torch.empty(n, nh, hd)
    for h in range(nh):
        s = (q[:, h] @ k[:, h // 2].T * 0.05).masked_fill(torch.ones(n, n).triu(1).bool(), float("-inf"))
        want[:, h] = (torch.softmax(s, dim=1) @ v[:, h // 2]).float()
    err = {}
    for exact in (0, 1):
        out = torch.full((n, nh * hd), 3e4, device="cuda")
        aa = K.AttnArgs()
        aa.q, aa.q_stride, aa.kv_new, aa.kv_stride = d.data_ptr(), d.stride(0), d.data_ptr() + nh * hd * 2, d.stride(0)
        aa.out, aa.out_stride, aa.out_f32, aa.exact_weights = out.data_ptr(), out.stride(0), 1, exact
        aa.cache, aa.batch, aa.nh, aa.nkv, aa.hd, aa.scale = view, ctx.layout.c_struct(), nh, nkv, hd, 0.05
        where = K.KV_FROM_STEP if source == "step" else K.KV_FROM_CACHE
        accepts, run = (K.attn_prefill_tc_accepts, K.attn_prefill_tc) if kernel == "tc" else (K.attn_prefill_mma_accepts, K.attn_prefill_mma)
        assert accepts(aa, torch.bfloat16, where)
        run(aa, where, ctx.stream)
        err[exact] = rel_l2(out.cpu(), want.reshape(n, -1))
    assert err[0] > 3e-4 and err[1] < 3e-5, err
    assert not K.wait_errors()


@pytest.mark.parametrize("hd,group", [(128, 6), (128, 16), (64, 4)])
def test_tensor_core_decode_of_pairs(hd, group):
    """Decode splits left in scratch and merged a pair of maps at a time, weights in two halves, against the any-size kernel on the
    same cache rows, at lengths inside a page, at its border and over many splits."""
    from titan_b200 import kernels as K
    from titan_b200.cache import SequenceCache
    from titan_b200.cache.groups import CacheNeed
    from titan_b200.engine.batch import StepEntry
    nkv, lens = 2, [1, 63, 64, 65, 700]
    nh, B = nkv * group, len(lens)
    g = torch.Generator().manual_seed(hd + group)
    cache = SequenceCache([CacheNeed("kv", nkv, hd)], 2048, B, 1024, torch.bfloat16, "cuda")
    slots = [cache.alloc_slot() for _ in lens]
    cache.reserve(dict(zip(slots, lens)))
    grp, index = cache.view_for_layer(0)
    view = K.KvView(grp.layer_storage(index).data_ptr(), grp.table.data_ptr(), grp.table_width, 0, grp.page_size, grp.num_pages, nkv, hd)
    fill = make_ctx([StepEntry(s, [0] * n, []) for s, n in zip(slots, lens)], [0] * B, torch.bfloat16)
    kv = torch.randn(sum(lens), 2 * nkv * hd, generator=g).to(torch.bfloat16).cuda()
    K.kv_append(kv, view, fill.layout.c_struct(), fill.stream)
    ctx = make_ctx([StepEntry(s, [0], []) for s in slots], [n - 1 for n in lens], torch.bfloat16)
    q = torch.randn(B, nh * hd, generator=g).to(torch.bfloat16).cuda()
    lam, width = torch.tensor([0.6], device="cuda"), hd - 8
    outs = []
    for fast, chunk, splits in ((True, 128, 4), (True, 64, 11), (False, 64, 11)):
        out = torch.empty(B, nh // 2 * width, dtype=torch.bfloat16, device="cuda")
        scratch = torch.full((B * nh * splits * (hd + 2),), float("nan"), device="cuda")
        aa = K.AttnArgs()
        aa.q, aa.q_stride, aa.out, aa.out_stride = q.data_ptr(), q.stride(0), out.data_ptr(), out.stride(0)
        aa.cache, aa.batch, aa.nh, aa.nkv, aa.hd, aa.scale = view, ctx.layout.c_struct(), nh, nkv, hd, 0.1
        aa.pair_lambda, aa.pair_eps, aa.pair_scale, aa.pair_width = lam.data_ptr(), 1e-5, 0.5, width
        aa.chunk, aa.n_splits, aa.scratch, aa.exact_weights = chunk, splits, scratch.data_ptr(), int(fast)
        if fast:
            assert K.attn_decode_mma_accepts(aa, torch.bfloat16)
            K.attn_decode_mma(aa, ctx.stream)
        else:
            K.attn_decode(aa, torch.bfloat16, ctx.stream)
        outs.append(out.float().cpu())
    for o in outs[:2]:
        rows_close(o, outs[2], "bfloat16", "pairs", slack=0.2)
    assert not K.wait_errors()


def latent_spec(H, dn, rd, dv, r, scale, base=10000.0, dims=None, eps=EPS):
    from titan_b200.config import MixerSpec, NormSpec, PositionSpec
    return MixerSpec("latent_attention", WIDTH, H, 1, dn, softmax_scale=scale, prefix="m.", position=PositionSpec("rope", dims or rd, base, "adjacent"),
                     extra=(("rot_dim", rd), ("value_dim", dv), ("kv_rank", r), ("latent_norm", NormSpec("rmsnorm", r, eps, "dkv.norm")),
                            ("sink", "sink"), ("out_gate", "g"), ("exact_weights", True)))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,dn,rd,dv,r,dims", [(3, 16, 8, 12, 20, None), (1, 5, 6, 9, 11, 4), (5, 12, 2, 4, 6, None), (2, 128, 64, 128, 64, None), (4, 32, 16, 48, 40, 10),
                                               (8, 24, 8, 16, 300, None)])
def test_latent_attention_with_a_sink_and_an_output_gate(dtype, H, dn, rd, dv, r, dims):
    """Sinks of a few units beside scores of about one, gates that open and close: whole prompts, portions, single tokens across a
    page's border, slots used again; the tensor-core sizes among them."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    mixer = MIXERS.build(latent_spec(H, dn, rd, dv, r, 0.3, base=500.0, dims=dims))
    w = weights_for(mixer, 31)
    w["m.sink"] = w["m.sink"] * 6
    w["m.g"] = w["m.g"] * 3
    bind(mixer, w, DT[dtype])
    m = latent(H, dn, rd, dv, r, 0.3, base=500.0, rot_dims=dims)
    lens = [150, 71]
    xs = inputs(lens, 32)
    want = [t64(P.latent_attention(x.numpy(), plain_weights(w, "m."), "", m, EPS)) for x in xs]
    cache = SequenceCache([mixer.cache_need()], 1024, 4, 512, DT[dtype], "cuda", mark_freed=True)
    for sizes in ([lens], [[60, 33], [50, 2], [2, 2], [2, 30]], [[1, 1]]):
        got = drive(mixer_step(mixer, cache), cache, xs, dtype, sizes)
        for i in range(2):
            rows_close(got[i], want[i], dtype, f"sequence {i}, portions {sizes}", row_factor=6.0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("sizes_of", [(16, 8, 16), (128, 64, 128)])
def test_a_sink_counts_once_however_the_keys_are_cut(dtype, sizes_of):
    """Queries and keys are zero, so every key weighs the same and a head's output is the mean value times n / (n + exp(sink)): a sink
    left out, counted once a split or scaled like a score changes the factor.  Sinks of log 200 (as much as all keys together), a
    tiny one and a huge one; in prompts (the tensor-core sizes too), portions and decoded."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    dn, rd, dv = sizes_of
    H, r, n = 3, 64, 200
    mixer = MIXERS.build(latent_spec(H, dn, rd, dv, r, 0.25))
    w = weights_for(mixer, 33)
    w["m.q"] = w["m.q"] * 0.0
    w["m.sink"] = torch.tensor([5.3125, -30.0, 12.0])
    w["m.g"] = w["m.g"] * 0.0                                      # gates of one half
    bind(mixer, w, DT[dtype])
    x = inputs([n], 34)[0]
    W = plain_weights(w, "m.")
    want = t64(P.latent_attention(x.numpy(), W, "", latent(H, dn, rd, dv, r, 0.25), EPS))
    c = P.rms_norm((x.numpy() @ W["dkv"].T)[:, :r], W["dkv.norm"], EPS)
    v = (c @ W["uv"].T).reshape(n, H, dv).mean(axis=0) * (n / (n + np.exp(np.array([5.3125, -30.0, 12.0]))))[:, None]
    assert rel_l2(t64(0.5 * v.reshape(-1) @ W["o"].T), want[-1]) < 1e-6
    cache = SequenceCache([mixer.cache_need()], 1024, 2, 512, DT[dtype], "cuda", mark_freed=True)
    for sizes in ([[n]], [[100], [2], [97]], [[n - 20]], [[1]]):
        rows_close(drive(mixer_step(mixer, cache), cache, [x], dtype, sizes)[0], want, dtype, f"portions {sizes}", row_factor=6.0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("dn,rd,dv,r", [(24, 8, 16, 24), (128, 64, 128, 128)])
@pytest.mark.parametrize("far", FAR)
def test_one_far_latent_decides(dtype, dn, rd, dv, r, far):
    """A head's query, moved into the latent space, points against the row's own latent, and the last input row is minus that at ``far``:
    that latent, among hundreds, takes nearly all the weight.  The scale is set so that its score is 60.  In a prompt, decoded, in
    portions, decoded from the key on."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    H, n = 2, LAST + 1
    x = inputs([n], 8)[0]
    x[-1] = -x[far]
    w = weights_for(MIXERS.build(latent_spec(H, dn, rd, dv, r, 1.0)), 7)
    w["m.sink"], w["m.dkv.norm"] = torch.tensor([0.5, -1.0]), torch.ones(r)
    w["m.dkv"][r:] = 0.0                                           # no rotated key part: the latents decide
    uk = w["m.uk"].reshape(H, dn, r).double()
    q = torch.zeros(H, dn + rd, WIDTH, dtype=torch.float64)
    q[:, :dn] = -torch.linalg.pinv(uk.transpose(1, 2)) @ w["m.dkv"][:r].double()
    w["m.q"] = q.reshape(H * (dn + rd), WIDTH).to(torch.bfloat16).float()
    W = plain_weights(w, "m.")
    c = P.rms_norm((x.numpy() @ W["dkv"].T)[:, :r], W["dkv.norm"], EPS)
    own = [(W["uk"].reshape(H, dn, r)[h] @ c[far]) @ (W["q"] @ x[-1].numpy()).reshape(H, dn + rd)[h, :dn] for h in range(H)]
    scale = float(60.0 / min(own))
    m = latent(H, dn, rd, dv, r, scale, base=1e6)
    mixer = MIXERS.build(latent_spec(H, dn, rd, dv, r, scale, base=1e6))
    bind(mixer, w, DT[dtype])
    want = t64(P.latent_attention(x.numpy(), W, "", m, EPS))
    alone = (W["uv"] @ c[far]) / (1 + np.exp(-(W["g"] @ x[-1].numpy())))
    assert rel_l2(t64(W["o"] @ alone), want[-1]) < 0.05, "the test's weights do not single the key out"
    cache = SequenceCache([mixer.cache_need()], 1024, 4, 512, DT[dtype], "cuda", mark_freed=True)
    through_every_cut(mixer_step(mixer, cache), cache, x, far, dtype, want)


# --------------------------------------------------------------------------- #
# whole models
# --------------------------------------------------------------------------- #
def close(got, want, dtype, what="", slack=2.0):
    """bfloat16: the unit norm of a difference of maps enlarges what rounding leaves of it, so the bound is twice a single part's."""
    rows_close(got, want, dtype, what, row_factor=6.0, slack=1.0 if dtype == "float32" else slack)


class World:
    """One small model: weights, plain logits of its requests, engines by dtype and options."""

    def __init__(self, name, seed, lengths):
        self.cfg = make_config(name)
        self.weights = random_weights(self.cfg, seed)
        self.numpy = as_numpy(self.weights)
        self.requests = [random_tokens(n, self.cfg["vocab"], 50 + i) for i, n in enumerate(lengths)]
        self._plain, self._engines = {}, {}

    def plain(self, tokens, layers=False):
        key = tuple(tokens)
        if key not in self._plain:
            after = []
            logits = P.forward(self.cfg, self.numpy, list(tokens), after_layer=lambda i, x: after.append(x.copy()))
            self._plain[key] = (t64(logits), t64(np.stack(after)))
        return self._plain[key][1 if layers else 0]

    def engine(self, dtype, **kw):
        from titan_b200 import Engine
        from titan_b200.config import config_from_dict
        key = (dtype, tuple(sorted(kw.items())))
        if key not in self._engines:
            opts = {"max_tokens": 1536, "max_slots": 6, "mark_freed_pages": True} | kw
            self._engines[key] = Engine.from_tensors(config_from_dict(self.cfg), self.weights, dtype=dtype, **opts)
        return self._engines[key]


LENGTHS = {"mix": [150, 9, 66, 1], "odd": [140, 64, 3, 129], "wide": [70, 200, 17, 2]}
_worlds = {}


def world(name):
    if name not in _worlds:
        _worlds[name] = World(name, {"mix": 1, "odd": 2, "wide": 3}[name], LENGTHS[name])
    return _worlds[name]


MODELS = [(n, d) for n in ("mix", "odd", "wide") for d in BOTH]


@pytest.mark.parametrize("name,dtype", MODELS)
def test_whole_prompts_and_the_residual_stream_after_every_layer(name, dtype):
    """Every prompt alone, logits at every position; layer by layer on the longest, so that the first layer that differs is named."""
    from titan_b200 import StepEntry
    wd = world(name)
    e = wd.engine(dtype)
    toks = max(wd.requests, key=len)
    seen = []
    e.layer_observer = lambda run, x: seen.append(x.clone())
    try:
        s = e.alloc_slot()
        e.step([StepEntry(s, toks, [0])])
        e.free_slot(s)
    finally:
        e.layer_observer = None
    want = wd.plain(toks, layers=True)
    assert len(seen) == len(want)
    for i, got in enumerate(seen):
        close(got, want[i], dtype, f"{name}: after layer {i}")
    for toks in wd.requests:
        close(run_in_pieces(e, toks, [len(toks)]), wd.plain(toks), dtype, f"{name}: prompt of {len(toks)}")
    e.check_kernels()
    e.cache.check()


@pytest.mark.parametrize("name,dtype", MODELS)
def test_prompt_then_token_by_token_and_portions_down_to_two(name, dtype):
    wd = world(name)
    e = wd.engine(dtype)
    toks = wd.requests[0]
    want = wd.plain(toks)
    close(run_in_pieces(e, toks, [len(toks) - 40]), want, dtype, f"{name}: prompt then 40 single tokens")
    close(run_in_pieces(e, toks, [1]), want, dtype, f"{name}: token by token from the first")
    close(run_in_pieces(e, toks, [64, 2, 2, 31, 1, 2, 40]), want, dtype, f"{name}: portions")
    close(run_in_pieces(e, toks, [2] * (len(toks) // 2)), want, dtype, f"{name}: portions of two")
    close(run_in_pieces(e, toks, [3, 61, 64, 1, 1, 9]), want, dtype, f"{name}: portions that end at a page's border")
    e.check_kernels()


@pytest.mark.parametrize("name,dtype", MODELS)
def test_a_batch_of_unequal_requests_against_each_alone_and_slots_used_again(name, dtype):
    """All requests as one batch of prompts, decoded together while the shorter ones leave; then the same again in the freed slots
    and pages (which were overwritten when they were freed), in the other order."""
    from titan_b200 import StepEntry
    wd = world(name)
    e = wd.engine(dtype)
    reqs = wd.requests
    tail = 6
    alone = [run_in_pieces(e, r, [max(1, len(r) - tail)]) for r in reqs]
    for turn in range(2):
        order = list(range(len(reqs))) if turn == 0 else list(reversed(range(len(reqs))))
        at = {i: max(1, len(reqs[i]) - tail) for i in order}
        slots = {i: e.alloc_slot() for i in order}
        got = {i: [] for i in order}
        out = e.step([StepEntry(slots[i], reqs[i][:at[i]], list(range(at[i]))) for i in order])
        o = 0
        for i in order:
            got[i].append(out[o:o + at[i]].float().cpu())
            o += at[i]
            if at[i] == len(reqs[i]):
                e.free_slot(slots[i])
        while any(at[i] < len(reqs[i]) for i in order):
            live = [i for i in order if at[i] < len(reqs[i])]
            out = e.step([StepEntry(slots[i], [reqs[i][at[i]]], [0]) for i in live])
            for k, i in enumerate(live):
                got[i].append(out[k:k + 1].float().cpu())
                at[i] += 1
                if at[i] == len(reqs[i]):
                    e.free_slot(slots[i])
        for i in order:
            close(torch.cat(got[i]), wd.plain(reqs[i]), dtype, f"{name}: request {i} in a batch, turn {turn}")
            close(torch.cat(got[i]), alone[i], dtype, f"{name}: request {i} in a batch against itself alone, turn {turn}")
        e.cache.check()
    e.check_kernels()


def test_sequences_at_prompts_and_at_single_tokens_in_one_step():
    """A step in which one sequence brings a prompt, one a portion and one a single token (the shift's state and its neighbour rows side by
    side in one launch), float32."""
    from titan_b200 import StepEntry
    wd = world("mix")
    e = wd.engine("float32")
    a, b, c = (random_tokens(n, wd.cfg["vocab"], 60 + n) for n in (40, 30, 25))
    sa, sb, sc = (e.alloc_slot() for _ in range(3))
    got = {"b": [e.step([StepEntry(sb, b[:12], list(range(12))), StepEntry(sc, c[:24], [])])[:12]]}
    out = e.step([StepEntry(sb, b[12:29], list(range(17))), StepEntry(sa, a[:39], list(range(39))), StepEntry(sc, c[24:], [0])])
    got["b"].append(out[:17])
    close(out[56:57], wd.plain(c)[24:25], "float32", "a single token beside prompts")
    out2 = e.step([StepEntry(sa, a[39:], [0]), StepEntry(sb, b[29:], [0])])
    close(torch.cat([out[17:56], out2[:1]]), wd.plain(a), "float32", "a prompt beside a portion")
    close(torch.cat(got["b"] + [out2[1:]]), wd.plain(b), "float32", "portions")
    for s in (sa, sb, sc):
        e.free_slot(s)
    e.cache.check()


@pytest.mark.parametrize("dtype", BOTH)
def test_a_shift_of_one_reads_the_previous_token_alone(dtype):
    """With shift factors of one and queries and keys of zero, a layer sees only the previous token's row: the last position's logits do
    not depend on anything else of its own than the residual stream, and a state that lost the last token of the step before
    gives another row.  Cut at every kind of place: a state of a prompt, of a portion of two, of a single token."""
    from titan_b200 import Engine
    from titan_b200.config import config_from_dict
    cfg = make_config("mix")
    w = random_weights(cfg, 6)
    for i in range(4):
        w[f"l{i}.shift"] = torch.ones_like(w[f"l{i}.shift"])
    toks = random_tokens(12, cfg["vocab"], 5)
    want = t64(P.forward(cfg, as_numpy(w), toks))
    for j in (3, 7, 8):
        other = list(toks)
        other[j] = (other[j] + 1) % cfg["vocab"]
        assert rel_l2(t64(P.forward(cfg, as_numpy(w), other))[j + 1], want[j + 1]) > 20 * TOL["float32"]
    e = Engine.from_tensors(config_from_dict(cfg), w, dtype=dtype, max_tokens=512, max_slots=2, mark_freed_pages=True)
    for sizes in ([12], [4, 2, 2, 1, 1, 2], [1], [11, 1], [2, 10]):
        close(run_in_pieces(e, toks, sizes), want, dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", BOTH)
def test_a_loud_first_token_reaches_far(dtype):
    """The first token's row is unlike the others': every later position feels it, through the first key and the first latent, in a
    prompt and when decoded token by token."""
    from titan_b200 import Engine
    from titan_b200.config import config_from_dict
    cfg = make_config("mix")
    w = random_weights(cfg, 5)
    w["embed"][3] *= 4
    toks = random_tokens(200, cfg["vocab"], 77)
    toks = [3] + [t if t != 3 else 5 for t in toks[1:]]
    want = t64(P.forward(cfg, as_numpy(w), toks))
    other = [4] + toks[1:]
    assert rel_l2(t64(P.forward(cfg, as_numpy(w), other))[-1], want[-1]) > 20 * TOL["float32"], "the first token does not reach the last position"
    e = Engine.from_tensors(config_from_dict(cfg), w, dtype=dtype, max_tokens=1024, max_slots=2)
    close(run_in_pieces(e, toks, [len(toks)]), want, dtype, "whole")
    close(run_in_pieces(e, toks, [100]), want, dtype, "decoded from 100")
    close(run_in_pieces(e, toks, [1, 2]), want, dtype, "decoded from the first tokens on")


@pytest.mark.parametrize("name,dtype", [("odd", "float32"), ("odd", "bfloat16"), ("wide", "bfloat16")])
def test_long_decoding(name, dtype):
    """A short prompt, then 400 single tokens over several pages."""
    wd = world(name)
    toks = random_tokens(420, wd.cfg["vocab"], 123)
    e = wd.engine(dtype)
    close(run_in_pieces(e, toks, [20]), wd.plain(toks), dtype, "long decoding")
    e.check_kernels()


@pytest.mark.parametrize("name", ["mix", "wide"])
def test_greedy_generation_through_the_scheduler(name):
    """Engine.generate (scheduler, sampler, captured decode steps) against greedy decoding with the plain implementation, in float32,
    where the argmax is decided."""
    from titan_b200.sampling import SamplerParams
    wd = world(name)
    e = wd.engine("float32", max_batch=3)
    prompts = [r[:12] for r in wd.requests if len(r) >= 12] + [wd.requests[-1]]
    steps = 10
    results = e.generate(prompts, max_tokens=steps, params=SamplerParams.greedy(), stop_tokens=())
    for p, r in zip(prompts, results):
        seq = list(p)
        for _ in range(steps):
            logits = t64(P.forward(wd.cfg, wd.numpy, seq)[-1])
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) < 1e-3:
                break                                           # a near tie: float32 and float64 may differ from here
            seq.append(int(logits.argmax()))
        n = len(seq) - len(p)
        assert n > 0 and list(r.tokens)[:n] == seq[len(p):], f"{name}: generation differs"
    e.cache.check()


@pytest.mark.parametrize("name", ["mix", "wide"])
def test_captured_decode_steps_give_the_whole_prompts_logits(name):
    """bfloat16, as served: a batch decoded through advance() (eager first, then replayed graphs) against whole prompts."""
    from titan_b200 import StepEntry
    from titan_b200.sampling import SamplerParams
    wd = world(name)
    e = wd.engine("bfloat16")
    prompts = [wd.requests[0][:40], max(wd.requests, key=len)[:90]]
    slots, toks = e.start(prompts, [SamplerParams.greedy()] * 2, [1, 2])
    seqs = [list(p) + [t] for p, t in zip(prompts, toks)]
    for _ in range(6):
        toks = e.advance(slots, [s[-1] for s in seqs])
        for s, t in zip(seqs, toks):
            s.append(t)
    captured = e.last_logits.float().cpu()
    for s in slots:
        e.finish(s)
    assert e.graph_launches > 0, "no decode step was replayed from a graph"
    fresh = [e.alloc_slot(), e.alloc_slot()]
    out = e.step([StepEntry(fresh[i], seqs[i][:-1], [len(seqs[i]) - 2]) for i in range(2)]).float().cpu()
    for s in fresh:
        e.free_slot(s)
    close(captured, out, "bfloat16", "captured against whole prompts")
    e.check_kernels()


@pytest.mark.parametrize("option", [dict(attention="plain"), dict(gemm="plain")])
def test_plain_kernels_give_the_same_logits(option):
    """The any-size attention and the CUDA-core products in bfloat16 where the tensor-core kernels would fit."""
    wd = world("wide")
    e = wd.engine("bfloat16", **option)
    toks = wd.requests[1]
    close(run_in_pieces(e, toks, [150]), wd.plain(toks), "bfloat16", str(option))


def test_trace_runner_as_a_subprocess(tmp_path):
    """bin/trace_run on a model folder: a batch of two prompts, single tokens after them while one request leaves, then many short
    requests at once, in slots and pages that were used before."""
    cfg = make_config("odd")
    weights = random_weights(cfg, 9)
    folder = write_folder(str(tmp_path / "model"), cfg, {k: v.to(torch.bfloat16) for k, v in weights.items()})
    a, b = random_tokens(70, cfg["vocab"], 1), random_tokens(21, cfg["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:60], "want": [0, 59]}, {"id": "b", "tokens": b[:20], "want": [19]}], "end": []}]
    for i in range(10):
        es = [{"id": "a", "tokens": [a[60 + i]], "want": [0]}]
        if i == 0:
            es.append({"id": "b", "tokens": [b[20]], "want": [0]})
        steps.append({"step": i + 1, "entries": es, "end": ["b"] if i == 0 else (["a"] if i == 9 else [])})
    many = [random_tokens(3, cfg["vocab"], 30 + i) for i in range(20)]
    steps.append({"step": 11, "entries": [{"id": f"m{i}", "tokens": m[:2], "want": []} for i, m in enumerate(many)], "end": []})
    steps.append({"step": 12, "entries": [{"id": f"m{i}", "tokens": m[2:], "want": [0]} for i, m in enumerate(many)], "end": [f"m{i}" for i in range(20)]})
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "192"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(13)]
    W = as_numpy(weights)
    pa, pb = t64(P.forward(cfg, W, a)), t64(P.forward(cfg, W, b))
    read = lambda name: torch.from_numpy(np.fromfile(out / name, dtype="<f4").reshape(-1, cfg["vocab"]))
    rows_close(read("0.f32"), torch.stack([pa[0], pa[59], pb[19]]), "float32", "step 0")
    rows_close(read("1.f32"), torch.stack([pa[60], pb[20]]), "float32", "step 1")
    rows_close(read("10.f32"), pa[69:70], "float32", "step 10")
    rows_close(read("12.f32"), torch.stack([t64(P.forward(cfg, W, m))[2] for m in many]), "float32", "twenty short requests")


def test_command_line_with_random_weights(tmp_path):
    """bin/titan_b200 run --random: the design through the command line, the scheduler and the sampler, from a description alone."""
    path = tmp_path / "config.json"
    path.write_text(json.dumps(make_config("mix")))
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "titan_b200"), "run", "--random", str(path), "--weights-seed", "3", "--prompt-ids", "5,6,7,8",
                        "--prompt-ids", "9,10", "--max-tokens", "12", "--temp", "0", "--dtype", "bfloat16", "--kv-capacity", "512"],
                       capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    assert p.stdout.strip(), "nothing was generated"


def drawn_config(seed):
    """A configuration drawn at random: sizes, head counts, layer order, readers, constants; odd sizes and ones included."""
    import random
    r = random.Random(seed)
    layers, owners = [], []
    for i in range(r.randint(1, 7)):
        ff = r.choice([None, 8, 17, 40, 64, 96])
        if r.random() < 0.5:
            if owners and r.random() < 0.5:
                src = r.choice(owners)
                o = layers[src]["mixer"]
                m = attention(o["heads"], o["kv_heads"], o["dim"], o["vdim"], r.choice([0.1, 0.3]), r.choice([0.0, 0.2, 0.7]), kv_from=src)
            else:
                kv, dim = r.choice([1, 2, 3]), r.choice([1, 4, 6, 8, 12, 16, 30, 32, 48, 64])
                m = attention(kv * r.choice([1, 2, 4]), kv, dim, r.choice([2 * dim, dim, 5, 24, 64]), r.choice([0.1, 0.3, dim ** -0.5]), r.choice([0.0, 0.2, 0.5, 0.8]))
                owners.append(i)
            layers.append(layer("attention", m, ff))
        else:
            rd = r.choice([2, 4, 8, 16])
            m = latent(r.choice([1, 2, 3, 4, 8]), r.choice([1, 4, 8, 12, 32]), rd, r.choice([1, 4, 8, 20, 48]), r.choice([3, 6, 16, 28, 72]), r.choice([0.1, 0.3]),
                       base=r.choice([100.0, 1e4, 5e5]), rot_dims=r.choice([d for d in (2, 4, 8, 16) if d <= rd]))
            layers.append(layer("latent_attention", m, ff))
    return model(layers, width=r.choice([24, 40, 51, 64, 96, 136]), vocab=r.choice([50, 97, 300]), eps=r.choice([1e-6, 1e-5, 1e-3]))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("seed", range(int(os.environ.get("PIPESUN_DRAWN", "12"))))
def test_configurations_drawn_at_random(seed, dtype):
    """A prompt whole, then a second request as a prompt with single tokens after it, in a batch with a third.  float32 is the sharp
    test (a wrong branch costs tens of percent, summation order 1e-6); bfloat16 by the rows' median and nine in ten, since a drawn
    model may hold a layer whose two maps nearly cancel."""
    from titan_b200 import Engine, StepEntry
    from titan_b200.config import config_from_dict
    cfg = drawn_config(seed)
    w = random_weights(cfg, 100 + seed)
    W = as_numpy(w)
    a, b, c = (random_tokens(n, cfg["vocab"], 7 * seed + n) for n in (75, 130, 9))
    e = Engine.from_tensors(config_from_dict(cfg), w, dtype=dtype, max_tokens=1024, max_slots=4, mark_freed_pages=True)
    whole = run_in_pieces(e, a, [len(a)])
    sb, sc = e.alloc_slot(), e.alloc_slot()
    got_b = [e.step([StepEntry(sb, b[:66], list(range(66))), StepEntry(sc, c[:8], [])])[:66]]
    got_b.append(e.step([StepEntry(sb, [b[66]], [0]), StepEntry(sc, [c[8]], [])])[:1])
    e.free_slot(sc)
    for t in b[67:]:
        got_b.append(e.step([StepEntry(sb, [t], [0])]))
    e.free_slot(sb)
    e.check_kernels()
    e.cache.check()
    for got, toks, what in ((whole, a, "whole"), (torch.cat(got_b).float().cpu(), b, "prompt in a batch, then single tokens")):
        want = t64(P.forward(cfg, W, toks))
        if dtype == "float32":
            rows_close(got, want, dtype, f"seed {seed}: {what}", row_factor=20.0, slack=2.0)
            continue
        rows = (got.double() - want.double()).norm(dim=1) / want.double().norm(dim=1)
        assert float(rows.median()) < 3 * TOL[dtype] and float((rows > 12 * TOL[dtype]).double().mean()) <= 0.1, f"seed {seed}: {what}: {float(rows.median()):.3f} {float(rows.max()):.3f}"


def test_a_steps_context_is_freed_with_its_last_reference():
    """Nothing of a step refers back to its context: the step's buffers go back to the allocator when the step returns, not when
    Python's cycle collector next runs (prompts would otherwise take new device memory step after step)."""
    import gc
    import weakref
    from titan_b200 import StepEntry
    wd = world("mix")
    e = wd.engine("bfloat16")
    made = []
    real = e._context
    e._context = lambda layout: (lambda ctx: (made.append(weakref.ref(ctx)), ctx)[1])(real(layout))
    was = gc.isenabled()
    gc.disable()
    try:
        s = e.alloc_slot()
        e.step([StepEntry(s, wd.requests[0], [0])])
        e.step([StepEntry(s, [1], [0])])
        e.free_slot(s)
        assert len(made) == 2 and all(r() is None for r in made), "a step's context outlives the step"
    finally:
        del e._context
        if was:
            gc.enable()

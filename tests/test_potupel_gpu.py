"""The Potupel design in the engine against the plain implementation (tests/plain/potupel_plain.py): every mechanism alone,
then whole models under every way of cutting the work.  Needs a B200; float32 (true 32-bit) and bfloat16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from helpers import TOL, random_tokens, rel_l2, rows_close, write_folder
from plain import potupel_plain as P
from potupel_cases import as_numpy, attention, dense, layer, make_config, model, moe, random_weights
from test_desalorn_gpu import BOTH, DT, WIDTH, bind, ctx_of, drive, inputs, make_ctx, mixer_step, plain_weights, run_in_pieces, t64, weights_for

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
EPS = 1e-5


# --------------------------------------------------------------------------- #
# mechanisms alone
# --------------------------------------------------------------------------- #
CONV_SIZES = [
    # heads, kv heads, head, taps, rotated, pairing
    (4, 2, 32, 3, 16, "half"),
    (6, 2, 64, 4, 64, "half"),              # the vector kernel's full window, the whole head rotated
    (2, 1, 128, 2, 32, "half"),
    (3, 3, 16, 1, 0, "half"),               # one tap: no window, no state; no rotation
    (1, 1, 256, 4, 128, "half"),
    (5, 1, 64, 4, 20, "adjacent"),
    (2, 2, 32, 3, 12, "half"),              # partners that are not whole vectors apart: the any-size kernel
    (3, 1, 48, 4, 16, "half"),              # heads that do not divide a warp's channels
    (2, 1, 16, 5, 8, "half"),               # longer windows
    (2, 1, 32, 9, 32, "adjacent"),
    (1, 1, 32, 40, 16, "half"),             # a window longer than most portions
]


@pytest.mark.parametrize("any_size", [False, True])
@pytest.mark.parametrize("H,G,hd,taps,rot,pairing", CONV_SIZES)
def test_convolution_rotation_and_append(H, G, hd, taps, rot, pairing, any_size):
    """Three unequal sequences in slots out of order: whole, in portions down to one token, token by token; queries, keys and values
    beside the cache, and the cache's own rows at the end (keys first, then values); the window's state after every step, other
    slots' states as they were.  Steps of single tokens also from float32 sums, which are left zeroed."""
    from titan_b200 import kernels as K
    from titan_b200.cache import SequenceCache
    from titan_b200.cache.groups import CacheNeed
    from titan_b200.config.spec import PositionSpec
    from titan_b200.engine.batch import StepEntry
    from titan_b200.parts import POSITIONS
    g = torch.Generator().manual_seed(hd + taps)
    C, Q, KV = (H + 2 * G) * hd, H * hd, G * hd
    w = torch.randn(C, taps, generator=g)
    lens = [75, 5, 12]
    scaling = (4.0, 1.0, 4.0, 64.0)
    position = POSITIONS.build(PositionSpec("rope", rot, 300.0, pairing, scaling) if rot else PositionSpec("none"))
    freq = P.frequencies(rot, 300.0, dict(zip(("factor", "low", "high", "original"), scaling)))
    for dtype in BOTH:
        xs = [torch.randn(n, C, generator=g).to(DT[dtype]) for n in lens]
        want = []
        for x in xs:
            y = P.causal_conv(x.double().numpy(), w.double().numpy())
            heads = y[:, :Q + KV].reshape(-1, H + G, hd)
            if pairing == "adjacent":        # the plain rotation pairs halves: bring the pairs' members there and back
                order = np.concatenate([np.arange(0, rot, 2), np.arange(1, rot, 2), np.arange(rot, hd)])
                turned = P.rotate_half(heads[..., order], np.arange(len(x)), freq)
                heads = np.empty_like(turned)
                heads[..., order] = turned
            else:
                heads = P.rotate_half(heads, np.arange(len(x)), freq)
            want.append(t64(np.concatenate([heads.reshape(-1, Q + KV), y[:, Q + KV:]], axis=1)))
        state = torch.full((6, max(1, taps - 1), C), 7.0, device="cuda")
        taps_d = w.t().contiguous().cuda()
        for plan in ([lens], [[20, 0, 5], [1, 2, 2], [2, 3, 0], [30, 0, 5], [22, 0, 0]], [[1, 1, 1]] * 75):
            cache = SequenceCache([CacheNeed("kv", G, hd)], 1024, 6, 256, DT[dtype], "cuda")
            taken = [cache.alloc_slot() for _ in range(5)]
            slots = [taken[4], taken[0], taken[2]]
            state[slots] = 0.0
            group, index = cache.view_for_layer(0)
            view = K.KvView(group.layer_storage(index).data_ptr(), group.table.data_ptr(), group.table_width, 0, group.page_size, group.num_pages, G, hd)
            at, got = [0, 0, 0], [[], [], []]
            for sizes in plan:
                take = [(i, min(n, lens[i] - at[i])) for i, n in enumerate(sizes) if n and at[i] < lens[i]]
                cache.reserve({slots[i]: at[i] + n for i, n in take})
                ctx = make_ctx([StepEntry(slots[i], [0] * n, []) for i, n in take], [at[i] for i, _ in take], DT[dtype])
                lay = ctx.layout
                x = torch.cat([xs[i][at[i]:at[i] + n] for i, n in take]).cuda()
                sums = lay.all_single
                if sums:
                    x = x.float()
                out = torch.full((x.shape[0], C), 3e4, dtype=DT[dtype], device="cuda")
                a = K.ConvQkvArgs()
                a.inp, a.in_stride, a.taps, a.n_taps = x.data_ptr(), C, taps_d.data_ptr(), taps
                if taps > 1:
                    a.state, a.state_stride = state.data_ptr(), state.stride(0)
                a.q_out, a.q_stride, a.kv_out, a.kv_stride = out.data_ptr(), C, out.data_ptr() + Q * out.element_size(), C
                a.rope, a.nh, a.nkv, a.hd = position.kernel_args("cuda"), H, G, hd
                a.q_start, a.start_pos, a.kv_len, a.slot_of_seq = lay.q_start.data_ptr(), lay.start_pos.data_ptr(), lay.kv_len.data_ptr(), lay.slot_of_seq.data_ptr()
                a.cache, a.append, a.zero_in, a.T, a.B, a.max_new = view, 1, int(sums), lay.T, lay.B, lay.max_new
                K.conv_qkv(a, x.dtype, out.dtype, ctx.stream, any_size=any_size)
                if sums:
                    assert float(x.abs().max()) == 0.0, "the sums were not left zeroed"
                o = 0
                for i, n in take:
                    got[i].append(out[o:o + n].float().cpu())
                    o, at[i] = o + n, at[i] + n
                    cache.commit(slots[i], at[i])
                    if taps > 1:
                        past = torch.cat([torch.zeros(taps - 1, C), xs[i][:at[i]].float()])[-(taps - 1):]
                        assert torch.equal(state[slots[i]].cpu(), past), f"state of sequence {i} at {at[i]}"
            for i in range(3):
                rows_close(torch.cat(got[i]), want[i], dtype, f"sequence {i}", row_factor=6.0)
                pages = group.pages_of[slots[i]]
                for plane, c0 in ((0, Q), (1, Q + KV)):
                    rows = group.layer_storage(index)[plane, pages].float().permute(0, 2, 1, 3).reshape(-1, KV)[:lens[i]]
                    rows_close(rows, want[i][:, c0:c0 + KV], dtype, f"cache plane {plane} of sequence {i}", row_factor=6.0)
            rest = [s for s in range(6) if s not in slots]
            assert bool((state[rest] == 7.0).all()), "a slot that is not in the batch was written"


def conv_spec(H, G, dim, vdim, scale, taps, rot, base=300.0, scaling=(4.0, 1.0, 4.0, 64.0), exact=True, window=None):
    from titan_b200.config import MixerSpec, PositionSpec
    return MixerSpec("attention", WIDTH, H, G, dim, softmax_scale=scale, prefix="a.", position=PositionSpec("rope", rot, base, "half", scaling), window=window,
                     names=tuple((r, r) for r in ("q", "k", "v", "o")),
                     extra=(("value_dim", vdim), ("conv", taps), ("sink_value", 0.0), ("exact_weights", exact)))


def plain_mixer(H, G, dim, vdim, scale, taps, rot, base=300.0, scaling=(4.0, 1.0, 4.0, 64.0)):
    return attention(H, G, dim, vdim, scale, taps, rot, base, scaling)


ATTENTION_SIZES = [
    (4, 2, 12, 20, 3, 8),                   # heads of 32, keys and values padded
    (3, 3, 7, 5, 4, 6),                     # as many kv heads as heads, no multiples of anything
    (2, 1, 3, 29, 5, 2),
    (1, 1, 16, 16, 1, 16),                  # one tap: no state beside the keys
    (6, 2, 64, 64, 4, 32),                  # tensor cores in bfloat16
    (9, 1, 60, 48, 2, 48),                  # padded to 64, nine heads on a kv head
    (2, 2, 128, 100, 3, 128),
    (4, 1, 100, 128, 4, 64),                # keys padded to 128
    (18, 1, 64, 40, 4, 24),                 # more heads on a kv head than the tensor-core decode kernel takes
    (2, 1, 40, 80, 2, 24),                  # heads of 80
    (2, 1, 200, 256, 3, 96),                # heads of 256
]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,dim,vdim,taps,rot", ATTENTION_SIZES)
def test_attention_behind_convolutions(dtype, H, G, dim, vdim, taps, rot):
    """Two unequal sequences, whole, in portions down to two tokens, single tokens across a page's border; then the slots again
    (freed pages overwritten)."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    scale = 2.0 * dim ** -0.5
    mixer = MIXERS.build(conv_spec(H, G, dim, vdim, scale, taps, rot))
    w = weights_for(mixer, 3)
    bind(mixer, w, DT[dtype])
    m = plain_mixer(H, G, dim, vdim, scale, taps, rot)
    xs = inputs([150, 71], 5)
    want = [t64(P.attention(x.numpy(), plain_weights(w, "a."), "", m)) for x in xs]
    cache = SequenceCache([mixer.cache_need()], 1024, 4, 512, DT[dtype], "cuda", mark_freed=True)
    for sizes in ([[150, 71]], [[60, 33], [50, 2], [2, 2], [2, 30]], [[2, 2]] * 12, [[1, 1]]):
        got = drive(mixer_step(mixer, cache), cache, xs, dtype, sizes)
        for i in range(2):
            rows_close(got[i], want[i], dtype, f"sequence {i}, portions {sizes[:4]}", row_factor=6.0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("window", [1, 20, 64, 70])
def test_convolutions_in_front_of_a_windowed_ring(dtype, window):
    """The same mixer over the last ``window`` keys only (no Potupel layer has a window; another design may): the ring takes a row
    only where no later token of the step does."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    H, G, dim, vdim, taps, rot = 4, 2, 16, 16, 3, 8
    mixer = MIXERS.build(conv_spec(H, G, dim, vdim, 0.5, taps, rot, window=window))
    w = weights_for(mixer, 3)
    bind(mixer, w, DT[dtype])
    W, m = plain_weights(w, "a."), plain_mixer(H, G, dim, vdim, 0.5, taps, rot)

    def windowed(x):
        T = x.shape[0]
        q, k, v = (P.causal_conv(x @ W[r].T, W[r + ".conv"]) for r in ("q", "k", "v"))
        freq = P.frequencies(rot, m["rot"]["base"], m["rot"]["scaling"])
        q, k = (P.rotate_half(a.reshape(T, -1, dim), np.arange(T), freq) for a in (q, k))
        out = np.empty((T, H, vdim))
        for h in range(H):
            s = q[:, h] @ k[:, h // 2].T * 0.5
            e = np.where(np.tril(np.ones((T, T))) - np.tril(np.ones((T, T)), -window) > 0, np.exp(s), 0.0)
            out[:, h] = e / (1.0 + e.sum(axis=1, keepdims=True)) @ v.reshape(T, G, vdim)[:, h // 2]
        return out.reshape(T, -1) @ W["o"].T
    xs = inputs([150, 71], 6)
    want = [t64(windowed(x.numpy())) for x in xs]
    cache = SequenceCache([mixer.cache_need()], 1024, 4, 512, DT[dtype], "cuda", mark_freed=True)
    for sizes in ([[150, 71]], [[60, 33], [50, 2], [2, 2], [2, 30]], [[1, 1]]):
        got = drive(mixer_step(mixer, cache), cache, xs, dtype, sizes)
        for i in range(2):
            rows_close(got[i], want[i], dtype, f"sequence {i}, portions {sizes}", row_factor=6.0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("dim", [16, 64, 128])
def test_one_in_the_denominator_counts_once_however_the_keys_are_cut(dtype, dim):
    """Queries are zero, so every score is 0 and the output at position t is the sum of the values over t + 2: an added one that is
    left out, counted once a split or scaled away changes the factor, most of all in the first tokens."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    H, G, n, taps = 4, 2, 200, 3
    mixer = MIXERS.build(conv_spec(H, G, dim, dim, 0.25, taps, 8))
    w = weights_for(mixer, 33)
    w["a.q"] = w["a.q"] * 0.0
    bind(mixer, w, DT[dtype])
    x = inputs([n], 34)[0]
    W = plain_weights(w, "a.")
    v = P.causal_conv(x.numpy() @ W["v"].T, W["v.conv"]).reshape(n, G, dim)
    mean = np.cumsum(v, axis=0) / (np.arange(n) + 2.0)[:, None, None]
    want = t64(np.repeat(mean, H // G, axis=1).reshape(n, -1) @ W["o"].T)
    assert rel_l2(want, t64(P.attention(x.numpy(), W, "", plain_mixer(H, G, dim, dim, 0.25, taps, 8)))) < 1e-6
    cache = SequenceCache([mixer.cache_need()], 1024, 2, 512, DT[dtype], "cuda", mark_freed=True)
    for sizes in ([[n]], [[100], [2], [97]], [[n - 20]], [[1]]):
        rows_close(drive(mixer_step(mixer, cache), cache, [x], dtype, sizes)[0], want, dtype, f"portions {sizes}", row_factor=6.0)


LAST = 229
FAR = [0, 1, 2, 63, 64, 65, 127, 128, 191, 192, LAST - 4]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("dim", [48, 64, 128])
@pytest.mark.parametrize("far", FAR)
def test_one_far_key_decides(dtype, dim, far):
    """The key matrix is the query matrix and the last input row is half of the one at ``far`` (the taps of q and k take
    the current token only): that key, among hundreds, takes nearly all the weight, and the
    last output is the value there, which the value's own taps gather from three tokens.  In a prompt, decoded, in portions."""
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    H, taps = 2, 3
    mixer = MIXERS.build(conv_spec(H, 1, dim, dim, 80.0 / dim, taps, 8, base=1e9, scaling=(1e6, 1.0, 4.0, 1e-3)))     # angles near zero: the rotation changes no score
    w = weights_for(mixer, 7)
    q = w["a.q"].reshape(H, dim, WIDTH)
    q[1] = q[0]
    w["a.q"], w["a.k"] = q.reshape(H * dim, WIDTH).contiguous(), q[0].clone()
    for r in ("q", "k"):
        w[f"a.{r}.conv"] = torch.zeros_like(w[f"a.{r}.conv"])
        w[f"a.{r}.conv"][:, -1] = 1.0
    bind(mixer, w, DT[dtype])
    m = plain_mixer(H, 1, dim, dim, 80.0 / dim, taps, 8, 1e9, (1e6, 1.0, 4.0, 1e-3))
    x = inputs([LAST + 1], 8)[0]
    x[far] *= 1.5                                                  # a loud row, and half of it: the far key beats the token's own
    x[far] = x[far].to(torch.bfloat16).double()
    x[-1] = x[far] * 0.5
    W = plain_weights(w, "a.")
    want = t64(P.attention(x.numpy(), W, "", m))
    v = P.causal_conv(x.numpy() @ W["v"].T, W["v.conv"])
    assert rel_l2(t64(np.tile(v[far], H) @ W["o"].T), want[-1]) < 0.2, "the test's weights do not single the key out"
    cache = SequenceCache([mixer.cache_need()], 1024, 4, 512, DT[dtype], "cuda", mark_freed=True)
    n = x.shape[0]
    for sizes, what in (([[n]], "in a prompt"), ([[n - 1]], "decoded alone"), ([[far + 1], [max(1, n - far - 3)], [2]], "in portions"), ([[max(1, far)]], "decoded from the key on")):
        rows_close(drive(mixer_step(mixer, cache), cache, [x], dtype, sizes)[0][-1:], want[-1:], dtype, what, row_factor=6.0)


@pytest.mark.parametrize("hd", [64, 128])
def test_the_tensor_core_kernels_are_asked_for_sixteen_bits_of_a_weight(hd, monkeypatch):
    """bfloat16 prompts, continued prompts and decode steps all run on tensor cores, with the weights in two halves."""
    from titan_b200 import kernels as K
    from titan_b200.cache import SequenceCache
    from titan_b200.parts import MIXERS
    asked = []
    for name in ("attn_prefill_tc", "attn_prefill_mma", "attn_decode_mma"):
        real = getattr(K, name)
        monkeypatch.setattr(K, name, lambda aa, *rest, real=real, name=name: (asked.append((name, aa.exact_weights)), real(aa, *rest))[1])
    mixer = MIXERS.build(conv_spec(4, 2, hd, hd, 0.1, 4, 16))
    bind(mixer, weights_for(mixer, 11), torch.bfloat16)
    cache = SequenceCache([mixer.cache_need()], 1024, 2, 512, torch.bfloat16, "cuda")
    drive(mixer_step(mixer, cache), cache, inputs([90], 12), "bfloat16", [[40], [48]])
    assert len(asked) == 4 and all(exact == 1 for _, exact in asked) and [n for n, _ in asked][2:] == ["attn_decode_mma"] * 2
    assert not K.wait_errors()


@pytest.mark.parametrize("M,N,Kd", [(1, 64, 48), (3, 33, 51), (8, 1000, 520), (9, 640, 256), (40, 1024, 512), (100, 96, 128), (130, 256, 64), (300, 1536, 512), (700, 200, 136), (2048, 3072, 1024)])
def test_squared_relu_in_the_products_epilogue(M, N, Kd):
    """max(z, 0)^2 of the float32 sum, rounded once: the rows, swapped, single-CTA and CTA-pair tensor-core kernels, the CUDA-core
    kernel; a plain store with the same sizes is as it was."""
    from titan_b200.parts import linear
    g = torch.Generator().manual_seed(M + N)
    x, w = (torch.randn(M, Kd, generator=g)).to(torch.bfloat16).float(), (torch.randn(N, Kd, generator=g) / Kd ** 0.5).to(torch.bfloat16).float()
    z = x.double() @ w.double().T
    from titan_b200 import kernels as K
    for dtype in BOTH:
        for options in ({}, {"gemm": "plain"}, {"small_products": False}):
            out = torch.empty(M, N, dtype=DT[dtype], device="cuda")
            for unary, want in ((K.UNARY_RELU2, z.clamp(min=0) ** 2), (K.UNARY_NONE, z)):
                linear.matmul(x.to(DT[dtype]).cuda(), w.to(DT[dtype]).cuda(), out, linear.EPI_STORE, ctx_of(M, dtype, options), unary=unary)
                err = float((out.double().cpu() - want).abs().max() / want.abs().max())
                assert err < (1e-5 if dtype == "float32" else 5e-3), f"{dtype} {options} activation {unary}: {err:.2e}"
    assert not K.wait_errors()


@pytest.mark.parametrize("E,top,T", [(1, 1, 5), (5, 2, 33), (8, 8, 7), (16, 4, 300), (100, 10, 64)])
def test_the_routers_bias_decides_and_weighs(E, top, T):
    """The bias joins the logits for the choice and for the softmax over the chosen ones."""
    from titan_b200 import kernels as K
    g = torch.Generator().manual_seed(E)
    z, b = torch.randn(T, E, generator=g), torch.randn(E, generator=g) * 2
    for bias in (b, None):
        ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
        K.moe_route(z.cuda(), E, top, False, ids, wts, None, K.current_stream(), bias=None if bias is None else bias.cuda())
        want_ids, want = P.route((z + (0 if bias is None else bias)).double().numpy(), top)
        assert ids.cpu().numpy().tolist() == want_ids.tolist()
        rows_close(wts, t64(want), "float32", "weights")


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("E,top,F,shared,T", [(5, 2, 24, 32, 9), (1, 1, 11, 9, 70), (6, 1, 64, None, 40), (8, 3, 64, 128, 300), (4, 4, 40, None, 200)])
def test_experts_with_a_router_bias(dtype, E, top, F, shared, T):
    """Few pairs, many pairs and whole prompts (three ways through the experts), with and without an expert for every token."""
    from titan_b200.config.spec import FeedForwardSpec
    from titan_b200.parts import FEED_FORWARDS
    W = 64
    part = FEED_FORWARDS.build(FeedForwardSpec("moe", W, F, prefix="f.", extra=(("experts", E), ("top", top), ("router_bias", True), ("shared_size", shared or 0),
                                                                             ("shared_gate", False))))
    w = weights_for(part, 5)
    w["f.router"] = w["f.router"] * 4
    w["f.router.b"] = torch.randn(E, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).float() * 2
    bind(part, w, DT[dtype])
    x = inputs([T], 3, W)[0]
    Wp = plain_weights(w, "f.")
    z = np.sort(x.numpy() @ Wp["router"].T + Wp["router.b"], axis=1)
    if top < E:                             # rows whose choice is no close call (the products' order of summation could turn one over)
        x = x[torch.from_numpy(z[:, -top] - z[:, -top - 1] > 1e-4)]
    want = t64(P.experts(x.numpy(), Wp, "", moe(E, top, F, shared)))
    out = torch.zeros(x.shape[0], W, device="cuda")
    part.forward(x.to(DT[dtype]).cuda(), ctx_of(x.shape[0], dtype), out)
    rows_close(out, want, dtype, "experts", row_factor=6.0)


@pytest.mark.parametrize("W,T", [(48, 3), (51, 9), (256, 1), (1000, 40), (4096, 5), (5000, 300)])
def test_entering_a_pass(W, T):
    """The stream beside the embedded rows through one matrix, plus the pass's own vector; either half alone."""
    from titan_b200 import kernels as K
    from titan_b200.config.spec import LoopSpec
    from titan_b200.parts.loop import LoopEntry
    g = torch.Generator().manual_seed(W)
    rnd = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
    x0, later = rnd(T, W), rnd(T, W) * 2
    wt = {"in": rnd(W, 2 * W) / W ** 0.5, "step": rnd(3, W)}
    Pw = {"loop.in": wt["in"].to(torch.bfloat16).double().numpy(), "loop.step": wt["step"].double().numpy()}
    d = lambda t: t.double().numpy()
    for dtype in BOTH:
        for mix, step in (("in", "step"), ("in", None), (None, "step")):
            entry = LoopEntry(LoopSpec(0, 1, 3, mix, step), W)
            bind(entry, {"in": wt["in"].to(torch.bfloat16).float(), "step": wt["step"]}, DT[dtype])
            ctx = ctx_of(T, dtype)
            x = x0.cuda().clone()
            entry.begin(x, ctx)
            assert torch.equal(x.cpu(), x0)
            state = x0
            for t in range(3):
                entry.enter(x, ctx, t)
                want = P.enter_pass(d(state), d(x0), Pw, t) if mix else d(state)
                if not step:
                    want = want - Pw["loop.step"][t]
                if not mix:
                    want = want + Pw["loop.step"][t]
                rows_close(x, t64(want), dtype, f"pass {t}, {mix}, {step}", row_factor=6.0)
                state = later
                x.copy_(later)
    out = torch.empty(T, W, dtype=torch.bfloat16, device="cuda")
    x = x0.cuda().clone()
    K.pass_entry(x, later.cuda(), wt["step"][1].cuda().contiguous(), out, K.current_stream())
    assert torch.equal(out.float().cpu(), x0) and torch.equal(x.cpu(), later + wt["step"][1])


@pytest.mark.parametrize("ff", [40, None])
@pytest.mark.parametrize("dtype", BOTH)
def test_scaled_norms_after_sublayers(dtype, ff):
    """A block against its equations, with norm weights around zero (some near minus one, where a factor vanishes) and scales of both
    signs and zero."""
    from titan_b200.cache import SequenceCache
    from titan_b200.config import config_from_dict
    from titan_b200.engine.batch import StepEntry
    from titan_b200.parts import build_block
    cfg = model([layer(attention(4, 2, 16, 16, 0.3, 3, 8), None if ff is None else dense(ff))], 56, 32, 1e-4)
    w = random_weights(cfg, 8)
    w["l0.norm1b"][:5] = -1.0
    w["l0.ls1"][5:9] = 0.0
    block = build_block(config_from_dict(cfg).to_model_spec().layers[0])
    bind(block, w, DT[dtype])
    x = torch.randn(50, 56, generator=torch.Generator().manual_seed(1)) * 2
    Pw = as_numpy(w)
    want = P.joined(x.double().numpy(), P.attention(P.rms_norm(x.double().numpy(), Pw["l0.norm1"], 1e-4), Pw, "l0.mix.", cfg["layers"][0]["mixer"]),
                    Pw["l0.norm1b"], Pw["l0.ls1"], 1e-4)
    if ff is not None:
        want = P.joined(want, P.dense(P.rms_norm(want, Pw["l0.norm2"], 1e-4), Pw, "l0.mlp."), Pw["l0.norm2b"], Pw["l0.ls2"], 1e-4)
    cache = SequenceCache([block.mixer.cache_need()], 256, 2, 128, DT[dtype], "cuda")
    s = cache.alloc_slot()
    cache.reserve({s: 50})
    ctx = make_ctx([StepEntry(s, [0] * 50, [])], [0], DT[dtype])
    got = x.cuda().clone()
    block.forward(got, ctx, cache.view_for_layer(0))
    rows_close(got, t64(want), dtype, "block", row_factor=6.0)
    if ff is None:
        assert torch.equal(got[:, :9].cpu(), x[:, :9]), "a factor of zero still adds something"


# --------------------------------------------------------------------------- #
# whole models
# --------------------------------------------------------------------------- #
ROUTED = ("mix", "odd", "routed")


def close(got, want, dtype, what="", routed=False):
    """bfloat16 with mixtures: a near tie between experts may turn over with rounding and change a whole row, so those models are
    judged by their rows' median and all but a few rows; float32 and models without mixtures, row by row."""
    if dtype == "float32" or not routed:
        return rows_close(got, want, dtype, what, row_factor=6.0, slack=1.0 if dtype == "float32" else 1.5)
    rows = (got.double().cpu() - want.double()).norm(dim=1) / want.double().norm(dim=1)
    bad = int((rows > 6 * TOL[dtype]).sum())
    assert float(rows.median()) < 1.5 * TOL[dtype] and bad <= max(1, 0.06 * len(rows)), f"{what}: median {float(rows.median()):.3f}, {bad} of {len(rows)} rows off"


class World:
    """One small model: weights, plain logits of its requests, engines by dtype and options."""

    def __init__(self, name, seed, lengths):
        self.name, self.cfg = name, make_config(name)
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

    def close(self, got, want, dtype, what):
        close(got, want, dtype, f"{self.name}: {what}", self.name in ROUTED)


LENGTHS = {"mix": [150, 9, 66, 1], "odd": [140, 64, 3, 129], "wide": [70, 200, 17, 2], "routed": [80, 180, 5, 1]}
_worlds = {}


def world(name):
    if name not in _worlds:
        _worlds[name] = World(name, {"mix": 1, "odd": 2, "wide": 3, "routed": 4}[name], LENGTHS[name])
    return _worlds[name]


MODELS = [(n, d) for n in LENGTHS for d in BOTH]


@pytest.mark.parametrize("name,dtype", MODELS)
def test_whole_prompts_and_the_residual_stream_after_every_run_of_a_layer(name, dtype):
    """Every prompt alone, logits at every position; run by run on the longest, so that the first layer or pass that differs is named."""
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
        wd.close(got, want[i], dtype, f"after run {i}")
    for toks in wd.requests:
        wd.close(run_in_pieces(e, toks, [len(toks)]), wd.plain(toks), dtype, f"prompt of {len(toks)}")
    e.check_kernels()
    e.cache.check()


@pytest.mark.parametrize("name,dtype", MODELS)
def test_prompt_then_token_by_token_and_portions_down_to_two(name, dtype):
    wd = world(name)
    e = wd.engine(dtype)
    toks = wd.requests[0]
    want = wd.plain(toks)
    wd.close(run_in_pieces(e, toks, [len(toks) - 40]), want, dtype, "prompt then 40 single tokens")
    wd.close(run_in_pieces(e, toks, [1]), want, dtype, "token by token from the first")
    wd.close(run_in_pieces(e, toks, [64, 2, 2, 31, 1, 2, 40]), want, dtype, "portions")
    wd.close(run_in_pieces(e, toks, [2] * (len(toks) // 2)), want, dtype, "portions of two")
    wd.close(run_in_pieces(e, toks, [3, 61, 64, 1, 1, 9]), want, dtype, "portions that end at a page's border")
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
            wd.close(torch.cat(got[i]), wd.plain(reqs[i]), dtype, f"request {i} in a batch, turn {turn}")
            wd.close(torch.cat(got[i]), alone[i], dtype, f"request {i} in a batch against itself alone, turn {turn}")
        e.cache.check()
    e.check_kernels()


@pytest.mark.parametrize("name", ["mix", "odd"])
def test_sequences_at_prompts_and_at_single_tokens_in_one_step(name):
    """A step in which one sequence brings a prompt, one a portion and one a single token (windows from states and from neighbour rows
    side by side in one launch), float32."""
    from titan_b200 import StepEntry
    wd = world(name)
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
@pytest.mark.parametrize("taps", [2, 3, 4, 7])
def test_the_oldest_tap_alone_reaches_back_to_one_token(dtype, taps):
    """Every channel passes its oldest tap only, so a position's queries, keys and values are those of the token taps - 1 before it, and
    zeros in the first ones: a window that is one short or one long, or a state that lost its oldest row, gives another row.  Cut
    at every kind of place."""
    from titan_b200 import Engine
    from titan_b200.config import config_from_dict
    cfg = model([layer(attention(4, 2, 16, 16, 0.4, taps, 8), dense(32)), layer(attention(2, 1, 12, 8, 0.4, taps, 4))], 48, 61, 1e-5, loop=(0, 1, 2))
    w = random_weights(cfg, 6)
    for k in w:
        if k.endswith(".conv"):
            w[k][:, 1:] = 0.0
    toks = random_tokens(20, 61, 5)
    want = t64(P.forward(cfg, as_numpy(w), toks))
    for other in (taps - 1, taps + 1):
        near = {k: v.clone() for k, v in w.items()}
        for k in near:
            if k.endswith(".conv"):
                near[k] = torch.nn.functional.pad(w[k], (1, 0))[:, :taps] if other < taps else torch.cat([w[k], torch.zeros(w[k].shape[0], 1)], dim=1)
        c = json.loads(json.dumps(cfg))
        for l in c["layers"]:
            l["mixer"]["conv"] = near["l0.mix.q.conv"].shape[1]
        assert rel_l2(t64(P.forward(c, as_numpy(near), toks)), want) > 20 * TOL["float32"]
    e = Engine.from_tensors(config_from_dict(cfg), w, dtype=dtype, max_tokens=512, max_slots=2, mark_freed_pages=True)
    for sizes in ([20], [4, 2, 2, 1, 1, 2, 8], [1], [11, 1, 2], [2, 10], [taps - 1, taps, 1]):
        close(run_in_pieces(e, toks, sizes), want, dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", BOTH)
def test_a_loud_first_token_reaches_far(dtype):
    """The first token's row is unlike the others': every later position feels it, in a prompt and when decoded token by token."""
    from titan_b200 import Engine
    from titan_b200.config import config_from_dict
    cfg = make_config("wide")
    w = random_weights(cfg, 5)
    w["embed"][3] *= 6
    toks = random_tokens(200, cfg["vocab"], 77)
    toks = [3] + [t if t != 3 else 5 for t in toks[1:]]
    want = t64(P.forward(cfg, as_numpy(w), toks))
    other = [4] + toks[1:]
    assert rel_l2(t64(P.forward(cfg, as_numpy(w), other))[-1], want[-1]) > 20 * TOL["float32"], "the first token does not reach the last position"
    e = Engine.from_tensors(config_from_dict(cfg), w, dtype=dtype, max_tokens=1024, max_slots=2)
    close(run_in_pieces(e, toks, [len(toks)]), want, dtype, "whole")
    close(run_in_pieces(e, toks, [100]), want, dtype, "decoded from 100")
    close(run_in_pieces(e, toks, [1, 2]), want, dtype, "decoded from the first tokens on")


@pytest.mark.parametrize("name,dtype", [("odd", "float32"), ("mix", "bfloat16"), ("wide", "bfloat16")])
def test_long_decoding(name, dtype):
    """A short prompt, then 400 single tokens over several pages."""
    wd = world(name)
    toks = random_tokens(420, wd.cfg["vocab"], 123)
    e = wd.engine(dtype)
    wd.close(run_in_pieces(e, toks, [20]), wd.plain(toks), dtype, "long decoding")
    e.check_kernels()


@pytest.mark.parametrize("name", ["mix", "wide", "routed"])
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


@pytest.mark.parametrize("name", ["wide", "routed"])
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
    wd.close(captured, out, "bfloat16", "captured against whole prompts")
    e.check_kernels()


@pytest.mark.parametrize("option", [dict(attention="plain"), dict(gemm="plain"), dict(reproducible=True)])
def test_other_kernels_give_the_same_logits(option):
    """The any-size attention, the CUDA-core products and products whose parts add up in order, in bfloat16."""
    wd = world("wide")
    e = wd.engine("bfloat16", **option)
    toks = wd.requests[1]
    wd.close(run_in_pieces(e, toks, [150]), wd.plain(toks), "bfloat16", str(option))


def test_trace_runner_as_a_subprocess(tmp_path):
    """bin/trace_run on a model folder: a batch of two prompts, single tokens after them while one request leaves, then many short
    requests at once, in slots and pages that were used before."""
    cfg = make_config("mix")
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
    close(read("0.f32"), torch.stack([pa[0], pa[59], pb[19]]), "float32", "step 0")
    close(read("1.f32"), torch.stack([pa[60], pb[20]]), "float32", "step 1")
    close(read("10.f32"), pa[69:70], "float32", "step 10")
    close(read("12.f32"), torch.stack([t64(P.forward(cfg, W, m))[2] for m in many]), "float32", "twenty short requests")


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
    """A configuration drawn at random: sizes, head counts, feed-forwards, loops, constants; odd sizes and ones included."""
    import random
    r = random.Random(seed)
    layers = []
    for _ in range(r.randint(1, 6)):
        kv, dim = r.choice([1, 2, 3]), r.choice([2, 4, 7, 8, 12, 16, 30, 32, 48, 64, 100, 128])
        scaling = r.choice([None, (r.choice([2.0, 8.0]), r.choice([0.5, 1.0]), r.choice([1.0, 4.0, 7.5]), r.choice([20, 100, 512]))])
        m = attention(kv * r.choice([1, 2, 4]), kv, dim, r.choice([1, 5, 8, 24, 64, 128, dim]), r.choice([0.1, 0.3, dim ** -0.5]), r.choice([1, 2, 3, 4, 4, 5, 8, 12]),
                      2 * r.randint(1, dim // 2), base=r.choice([50.0, 1e4, 5e5]), scaling=scaling)
        E = r.choice([1, 2, 5, 8])
        layers.append(layer(m, r.choice([None, dense(r.choice([8, 17, 64])), moe(E, r.randint(1, E), r.choice([8, 13, 40]), r.choice([None, 6, 32]))])))
    loop = None
    if r.random() < 0.7:
        start = r.randrange(len(layers))
        loop = (start, r.randint(start + 1, len(layers)), r.choice([1, 2, 3]))
    return model(layers, width=r.choice([24, 40, 51, 64, 96, 136]), vocab=r.choice([50, 97, 300]), eps=r.choice([1e-6, 1e-5, 1e-3]), loop=loop)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("seed", range(int(os.environ.get("POTUPEL_DRAWN", "12"))))
def test_configurations_drawn_at_random(seed, dtype):
    """A prompt whole, then a second request as a prompt with single tokens after it, in a batch with a third.  float32 is the sharp
    test (a wrong branch costs tens of percent, summation order 1e-6); bfloat16 by the rows' median and nine in ten."""
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

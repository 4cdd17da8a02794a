"""Differential attention as a mixer: two softmax maps a head over the same values, one taken off the other.

    q = W_q h + b_q  (heads x 2 x dim);   k = W_k h + b_k  (kv heads x 2 x dim);   v = W_v h + b_v  (kv heads x value_dim)
    q, k <- rms over dim, a weight of dim shared by all heads and maps      (``qk_norm``)
    a_m  = softmax over keys j <= i of (q_m . k_m * scale), times v          m = 1, 2
    l    = exp(sum(lq1 * lk1)) - exp(sum(lq2 * lk2)) + diff                  one number for the layer
    o    = (a_1 - l a_2) / rms(a_1 - l a_2) * (1 - diff);   out += [o of every head] . W_o^T

The two maps of a head are two query heads of one kv head for every attention kernel: a kv head's cached key row is
[k of map 1 | k of map 2 | zeros] and its value row [v | zeros], both ``hd`` wide (the larger of 2 dim and value_dim, rounded up to
16), and a map's query lies over the same elements with zeros where the other map's key is.  So a value is stored and read
once for both maps, the cache is the ``kv`` group of grouped-query attention, and its kernels run as they are.  Between the
projections (one float32 product) and the attention, ``pair_prep`` adds the biases, norms, lays the rows out and appends; the
difference and its norm are float32 inside the kernel that finishes the softmax (the merge of decode splits, the any-size
prompt kernel) or, behind the tensor-core prompt kernels, which leave float32 rows, in ``pair_combine``.  The tensor-core
kernels keep sixteen bits of a softmax weight in its product with the values (``exact_weights``).

With ``cache_from`` the mixer owns no keys: it projects queries only and reads the named layer's cache.

Options (``MixerSpec.extra``): ``value_dim``, ``diff``, ``out_eps`` (the eps of the unit norm on a head's difference), ``bias`` (q, k
and v have biases, tensors ``<name>.b``).  Tensor names by role: q, k, v, o, lq1, lk1, lq2, lk2; the head norm's weight is
``qk_norm.weight`` with "q" or "k" put in (None: no norm).
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from .. import kernels as K
from ..cache.groups import CacheNeed, KVGroup
from ..weights.loader import WeightSpec
from . import linear
from .attention import decode_split
from .base import MIXERS, Mixer
from .norm import rows_of


class DifferentialAttentionMixer(Mixer):
    def __init__(self, spec):
        s = spec
        self.spec = s
        self.H, self.G, self.dim, self.dv = s.num_heads, s.num_kv_heads, s.head_dim, int(s.option("value_dim", 2 * s.head_dim))
        if self.H <= 0 or self.G <= 0 or self.H % self.G:
            raise ValueError(f"{self.H} query heads are not a multiple of {self.G} kv heads")
        if self.dim <= 0 or self.dv <= 0:
            raise ValueError("differential attention needs positive dim and value_dim")
        self.hd = -(-max(2 * self.dim, self.dv) // 16) * 16            # the one width keys (both maps) and values are stored at
        if self.hd > 1024:
            raise ValueError(f"two maps of {self.dim} and values of {self.dv}: rows of up to 1024 elements are supported")
        if s.window is not None or s.position.kind != "none":
            raise ValueError("differential attention comes without a window and without a rotation")
        self.shared = s.cache_from is not None
        self.diff, self.out_eps = float(s.option("diff", 0.0)), float(s.option("out_eps", 1e-6))
        if not self.out_eps > 0:
            raise ValueError("out_eps must be positive")
        self.has_bias = bool(s.option("bias", False))
        self.scale = s.softmax_scale if s.softmax_scale is not None else 1.0 / math.sqrt(self.dim)
        self.w_in = self.w_o = self.bias = self.q_norm = self.k_norm = self.lam = None
        self._views = {}

    # -- declaration ------------------------------------------------------ #
    def cache_need(self) -> Optional[CacheNeed]:
        return None if self.shared else CacheNeed("kv", self.G, self.hd)

    def _name(self, role: str) -> str:
        return self.spec.name(role, role)

    def _projections(self):
        """(role, rows) of the projections this layer owns, in the order of the fused product's columns."""
        own = [("q", 2 * self.H * self.dim)]
        return own if self.shared else own + [("k", 2 * self.G * self.dim), ("v", self.G * self.dv)]

    def weight_specs(self, prefix: str) -> List[WeightSpec]:
        s, p = self.spec, prefix + self.spec.prefix
        specs = [WeightSpec(p + self._name(r), (n, s.hidden_size)) for r, n in self._projections()]
        if self.has_bias:
            specs += [WeightSpec(p + self._name(r) + ".b", (n,), "vector", ("normal", 0.1)) for r, n in self._projections()]
        if s.qk_norm is not None:
            specs += [WeightSpec(p + s.qk_norm.weight.format(r), (self.dim,), "vector", ("one_plus_normal", 0.1)) for r in (("q",) if self.shared else ("q", "k"))]
        specs += [WeightSpec(p + self._name(r), (self.dim,), "vector", ("normal", 0.1)) for r in ("lq1", "lk1", "lq2", "lk2")]
        return specs + [WeightSpec(p + self._name("o"), (s.hidden_size, self.H * self.dv))]

    def bind(self, get) -> None:
        s, p = self.spec, self.spec.prefix
        parts = [get(p + self._name(r)) for r, _ in self._projections()]
        self.w_in = torch.cat(parts, dim=0).contiguous() if len(parts) > 1 else parts[0]
        if self.has_bias:
            self.bias = torch.cat([get(p + self._name(r) + ".b").float() for r, _ in self._projections()]).contiguous()
        if s.qk_norm is not None:
            self.q_norm = get(p + s.qk_norm.weight.format("q")).contiguous()
            self.k_norm = None if self.shared else get(p + s.qk_norm.weight.format("k")).contiguous()
        l = {r: get(p + self._name(r)).float() for r in ("lq1", "lk1", "lq2", "lk2")}
        lam = torch.exp((l["lq1"] * l["lk1"]).sum()) - torch.exp((l["lq2"] * l["lk2"]).sum()) + self.diff
        self.lam = lam.reshape(1).contiguous()                          # float32, once: it depends on weights alone
        self.w_o = get(p + self._name("o"))

    # -- one step --------------------------------------------------------- #
    def _view(self, cache) -> K.KvView:
        group, index = cache
        key = (id(group), index)
        if key not in self._views:
            if not isinstance(group, KVGroup) or group.need.head_dim != self.hd or group.need.num_kv_heads != self.G:
                raise TypeError(f"differential attention reads {self.G} heads of {self.hd} from a 'kv' cache group, not from {type(group).__name__}")
            self._views[key] = K.KvView(group.layer_storage(index).data_ptr(), group.table.data_ptr(), group.table_width,
                                        group.ring_rows, group.page_size, group.num_pages, group.need.num_kv_heads, group.need.head_dim)
        return self._views[key]

    def forward(self, h, ctx, cache, out: torch.Tensor) -> None:
        s, lay = self.spec, ctx.layout
        T, H, G, hd, dv = lay.T, self.H, self.G, self.hd, self.dv
        view = self._view(cache)
        decode = lay.all_single
        proj = ctx.empty((T, self.w_in.shape[0]), torch.float32)
        linear.matmul(rows_of(h), self.w_in, proj, linear.EPI_F32, ctx)
        Q, KV = 2 * H * hd, (0 if self.shared else G * hd)
        rows = ctx.empty((T, Q if decode else Q + 2 * KV))              # queries | the step's own keys | values
        pa = K.PairPrepArgs()
        pa.inp, pa.in_stride = proj.data_ptr(), proj.stride(0)
        pa.bias = None if self.bias is None else self.bias.data_ptr()
        pa.q_w = None if self.q_norm is None else self.q_norm.data_ptr()
        pa.k_w = None if self.k_norm is None else self.k_norm.data_ptr()
        pa.eps = s.qk_norm.eps if s.qk_norm is not None else 0.0
        pa.q_out, pa.q_stride = rows.data_ptr(), rows.stride(0)
        if not decode and not self.shared:
            pa.kv_out, pa.kv_stride = rows.data_ptr() + Q * rows.element_size(), rows.stride(0)
        pa.H, pa.G, pa.dim, pa.vdim, pa.hd = H, (0 if self.shared else G), self.dim, dv, hd
        pa.pos_of, pa.seq_of, pa.slot_of_seq = lay.pos_of.data_ptr(), lay.seq_of.data_ptr(), lay.slot_of_seq.data_ptr()
        # the cache keeps every key, so a row of the step replaces none that a query still reads: always appended at once
        pa.cache, pa.append, pa.T = view, int(not self.shared), T
        K.pair_prep(pa, ctx.dtype, ctx.stream)

        o = ctx.empty((T, H * dv))
        aa = K.AttnArgs()
        aa.q, aa.q_stride = rows.data_ptr(), rows.stride(0)
        aa.cache, aa.batch = view, lay.c_struct()
        aa.nh, aa.nkv, aa.hd, aa.scale = 2 * H, G, hd, self.scale
        tensor = ctx.options.get("attention", "fast") != "plain" and ctx.dtype == torch.bfloat16 and hd in (64, 128)
        aa.exact_weights = int(tensor and bool(ctx.options.get("exact_weights", True)))
        if decode:
            self._pair(aa, o)
            fast = tensor and K.attn_decode_mma_accepts(self._split(aa, ctx, True), ctx.dtype)
            if fast:
                if ctx.options.get("early_pages", True):       # lengths the kernel may read before its predecessors end
                    if lay.lengths_by_copy:
                        aa.early_len, aa.early_mode = lay.kv_len.data_ptr(), 1
                    elif lay.committed_len is not None:
                        aa.early_len, aa.early_mode = lay.committed_len.data_ptr(), 2
                K.attn_decode_mma(aa, ctx.stream)
            else:
                K.attn_decode(self._split(aa, ctx, False), ctx.dtype, ctx.stream)
        else:
            if not self.shared:
                aa.kv_new, aa.kv_stride = rows.data_ptr() + Q * rows.element_size(), rows.stride(0)
            if tensor:
                maps = ctx.empty((T, 2 * H * hd), torch.float32)
                aa.out, aa.out_stride, aa.out_f32 = maps.data_ptr(), maps.stride(0), 1
                source = K.KV_FROM_STEP if lay.all_fresh and not self.shared else K.KV_FROM_CACHE
                mode = ctx.options.get("attention", "fast")
                if mode == "fast" and K.attn_prefill_tc_accepts(aa, ctx.dtype, source):
                    K.attn_prefill_tc(aa, source, ctx.stream)
                elif K.attn_prefill_mma_accepts(aa, ctx.dtype, source):
                    K.attn_prefill_mma(aa, source, ctx.stream)
                else:
                    tensor = False
            if tensor:
                K.pair_combine(maps, hd, self.lam, o, dv, self.out_eps, 1.0 - self.diff, ctx.stream)
            else:
                aa.out_f32 = 0
                self._pair(aa, o)
                K.attn_prefill(aa, ctx.dtype, ctx.stream)
        linear.matmul(o, self.w_o, out, linear.EPI_ADD, ctx)

    def _pair(self, aa: K.AttnArgs, o: torch.Tensor) -> None:
        aa.out, aa.out_stride = o.data_ptr(), o.stride(0)
        aa.pair_lambda, aa.pair_eps, aa.pair_scale, aa.pair_width = self.lam.data_ptr(), self.out_eps, 1.0 - self.diff, self.dv

    def _split(self, aa: K.AttnArgs, ctx, fast: bool) -> K.AttnArgs:
        """Splits and scratch of a decode step for the tensor-core or the any-size kernel."""
        lay = ctx.layout
        options = ctx.options
        if not fast:
            # one block takes a kv head's maps in turns of four: more blocks where that leaves SMs idle, and shorter splits for few sequences
            group = 2 * self.H // self.G
            aa.head_blocks = self.G * (group // 4) if group % 4 == 0 else (self.G * (group // 2) if group % 2 == 0 else 2 * self.H)
            few = lay.B * aa.head_blocks * -(-lay.max_kv_len // 128) < int(options.get("sm_count", 148))
            options = dict(options, attn_chunk=int(options.get("pair_chunk", 64 if few else 128)))
        aa.chunk, aa.n_splits = decode_split(lay, self.G, options, fast)
        need = lay.B * 2 * self.H * aa.n_splits * (self.hd + 2)
        scratch = ctx.scratch.get("attn_partials")
        if scratch is None or scratch.numel() < need:
            scratch = ctx.scratch["attn_partials"] = torch.empty(need, dtype=torch.float32, device=ctx.device)
        aa.scratch = scratch.data_ptr()
        return aa


MIXERS.register("differential_attention", DifferentialAttentionMixer)

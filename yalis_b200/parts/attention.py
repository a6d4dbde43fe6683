"""Grouped-query causal attention over the paged cache.

qkv = x Wqkv^T; positions are encoded into Q and K and K, V stored (the position
part does both in one kernel); every token attends to the cached keys of its
request up to its own position; the heads are projected back with Wo
(yalis/external/model.py:540-608).  The three projections are stored
concatenated [Wq; Wk; Wv] (the reference interleaves them per KV group,
model.py:544-557, which only serves its tensor-parallel split).
"""

from __future__ import annotations

import math
from fractions import Fraction
from typing import Dict, Optional

import torch

from yalis_b200.config.spec import PartSpec
from yalis_b200.ops import attention as attn_ops
from yalis_b200.ops.linear import linear_partial
from yalis_b200.ops.elementwise import qkv_prepare
from .base import NOT_ROTARY, Mixer, NormedSum, PagedKV, PagedKVCache, ParamSpec, PositionEncoding, Projected, register_part


class PagedAttention(Mixer):
    """Parameters: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``,
    ``window`` (None = all keys), ``scale`` (None = 1/sqrt(head_dim))."""

    def __init__(self, spec: PartSpec, position: Optional[PositionEncoding] = None):
        super().__init__(spec, position)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.nh = int(p["num_heads"])
        self.g = int(p["num_kv_heads"])
        self.hs = int(p["head_dim"])
        self.window = p.get("window")
        self.scale = float(p["scale"]) if p.get("scale") is not None else 1.0 / math.sqrt(self.hs)
        if self.nh % self.g:
            raise ValueError(f"num_heads {self.nh} is not a multiple of num_kv_heads {self.g}")
        if self.hs % 2 or self.hs > 256:
            raise ValueError(f"head_dim {self.hs} is not supported (even, at most 256)")
        if position is None:
            raise ValueError("paged_attention needs a position part (use kind 'none' for no encoding)")
        self.w_qkv: Optional[torch.Tensor] = None
        self.w_o: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {
            "q_proj": ParamSpec((self.nh * self.hs, self.hidden)),
            "k_proj": ParamSpec((self.g * self.hs, self.hidden)),
            "v_proj": ParamSpec((self.g * self.hs, self.hidden)),
            "o_proj": ParamSpec((self.hidden, self.nh * self.hs)),
        }

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_qkv = torch.cat([tensors["q_proj"], tensors["k_proj"], tensors["v_proj"]], dim=0).contiguous()
        self.w_o = tensors["o_proj"].contiguous()

    def cache_request(self) -> PagedKV:
        return PagedKV(self.g, self.hs, self.window)

    def capture_key(self, host):
        # everything the choice of kernel and its launch depend on besides the shapes of the step's tensors
        per = self.nh // self.g
        if host.max_q_len == 1:
            return host.once(("decode_step_kind",), lambda: attn_ops.decode_step_kind([b + 1 for b in host.ctx_before]))
        return host.once(("portion_step_kind", per, self.g, self.hs),
                         lambda: attn_ops.portion_step_kind(host, per, self.g, self.hs))

    def mixing_flops(self, q_len: int, ctx_before: int) -> float:
        # QK^T and PV over the keys each token sees (causal; a window bounds them)
        keys = sum(min(ctx_before + t + 1, self.window or (ctx_before + t + 1)) for t in range(q_len)) if self.window \
            else q_len * ctx_before + q_len * (q_len + 1) / 2
        return 4.0 * self.nh * self.hs * keys

    def forward(self, x: torch.Tensor, ctx, cache: PagedKVCache) -> torch.Tensor:
        qkv = linear_partial(x, self.w_qkv)          # [N, width], or float32 partial sums [S, N, width]
        if (attn_ops.USE_FUSED_ROPE and ctx.n_requests * self.g <= 2 * attn_ops.sm_count(x.device)
                and attn_ops.decode_tma_applicable(x.dtype, ctx, self.hs, cache.k.shape[2], self.nh // self.g, self.window)
                and not attn_ops.decode_lean_preferred(ctx.n_requests, self.g, self.hs, attn_ops.step_kind(ctx)[0])):
            # A decode step whose attention blocks fit the GPU at once: the attention kernel rotates Q and the new K
            # itself and stores K, V (one launch less).  With more blocks than that the extra work at the start of
            # every block costs more than the launch (measured at batch 64: 59.5 against 57 us per layer).
            freq = self.position.rotary_frequencies(self.hs, x.device)
            if freq is not NOT_ROTARY:
                y = attn_ops.decode_attention_tma_fused(
                    qkv, freq, cache.writable, cache.k, cache.v, ctx.positions, ctx.q_start,
                    ctx.block_tables[cache.group], self.nh, self.g, self.hs, scale=self.scale,
                    n_splits=attn_ops.decode_tma_splits(ctx.n_requests, self.g, attn_ops.step_kind(ctx)[1]),
                    error_flag=ctx.error_flag,
                    early_fetch=bool(getattr(ctx, "settled", False)))
                return linear_partial(y, self.w_o)
        q = self.position.encode_and_store(qkv, self.nh, self.g, self.hs, ctx, cache, dtype=x.dtype)
        y = attn_ops.paged_attention(q, cache.k, cache.v, ctx, cache.group, self.nh, self.g, self.hs,
                                     scale=self.scale, window=self.window)
        return linear_partial(y, self.w_o)             # the residual stream adds the partial sums


def distance_bucket(n: int, buckets: int, far: float) -> int:
    """Which of ``buckets`` = B learned numbers the distance n >= 0 takes: n itself below h = B / 2, from there on
    h + floor(ln(n / h) / ln(far / h) * (B - h)), at most B - 1.  The floor is taken exactly: it is at least k when
    (n / h)^(B - h) >= (far / h)^k, a comparison of rational numbers (a logarithm in floating point falls short of whole
    results now and then, ln(2) / ln(32) * 5 for one)."""
    if buckets < 2 or buckets % 2:
        raise ValueError(f"a bias per distance needs an even number of buckets, not {buckets}")
    h = buckets // 2
    if not far > h:
        raise ValueError(f"the largest distance with a bucket of its own, {far}, must lie beyond {h}")
    if n < h:
        return n
    grown, step = Fraction(n, h) ** (buckets - h), Fraction(far) / h
    k, power = 0, step
    while h + k < buckets - 1 and grown >= power:
        k, power = k + 1, power * step
    return h + k


def distance_reach(buckets: int, far: float) -> int:
    """The smallest L such that all distances from L - 1 on share a bucket, the last."""
    lo, hi = 0, max(1, math.ceil(far))
    while lo < hi:                           # buckets grow with the distance
        mid = (lo + hi) // 2
        lo, hi = (lo, mid) if distance_bucket(mid, buckets, far) == buckets - 1 else (mid + 1, hi)
    return lo + 1


class GeneralAttention(Mixer, Projected):
    """Grouped-query causal attention over the paged cache with the variations that the fast kernels of
    ``paged_attention`` do not take.  Parameters: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``
    (of q and k), ``v_head_dim`` (None: head_dim), ``bias`` (q, k, v = W x + b), ``qk_norm_eps`` (None: no norm;
    else q and k of every head become x / sqrt(mean(x^2) + eps) * scale before the rotation, one learned scale
    [head_dim] for q and one for k), ``qk_norm_over`` (``head``, the default, or ``all``: the mean is over all heads of q,
    and of k, at once, the learned scales are [heads * head_dim]), ``qk_norm_weight`` (False: a norm without learned
    scales), ``values_from_keys`` (the values are the keys as projected, before their norm and rotation: no value matrix),
    ``rotary`` ({"dims", "theta", "layout", "scaling"}: the first ``dims`` sizes of a head turn, size i paired with
    i + dims / 2, or with layout ``interleaved`` size 2i with 2i + 1; ``scaling`` as the rotary part takes it, YaRN's
    factor on cosine and sine included; None: no rotation), ``scale``
    (None: 1/sqrt(head_dim)), ``softcap`` (c: scores become c tanh(s / c)), ``sink`` (True: 1 is added to the
    softmax's denominator; ``"learned"``: exp(z_h) with a learned z per head, the tensor ``sink``), ``window`` (position
    p sees the W positions up to itself), ``chunk`` (position p sees only its own chunk of C positions, counted from
    position 0, up to itself), ``distance_slopes`` (one number per head: slope_h * (p - j) is taken off the scaled
    score of key j), ``distance_bias`` ({"buckets": B, "max": D}: rel[bucket(p - j), h] with a learned table ``rel``
    [B, heads] is added to the scaled score, see ``distance_bucket``), ``pool`` (P, with a window: beside the window's
    keys position p sees one key and one value for every block of P positions, counted from position 0, that lies wholly
    before the window: the means of the block's keys and values as the cache holds them; tokens and blocks share one
    softmax), ``q_temperature`` ({"coef", "every"}: the query at position p is multiplied by
    1 + coef ln(floor((p + 1) / every) + 1)), ``gate`` (the heads' results are multiplied by sigmoid(W_g x), one more
    matrix over the mixer's input; ``"head"``: one number per head instead of one per element), ``difference`` ({"offset":
    d, "eps"}: two maps per head over the same values: q and k have two parts of ``head_dim`` sizes per head, side by side,
    each with the norm and rotation of a head of its own; each pair of parts is an attention of its own, and of the maps'
    results a1 and a2 the head's is (1 - d) o / sqrt(mean(o^2) + eps) with o = a1 - b a2 and b = exp(lq1 . lk1) -
    exp(lq2 . lk2) + d, one number for the layer from the learned vectors ``lq1`` ... ``lk2`` [head_dim]),
    ``out_bias`` (a bias on the output product), ``own_kv`` (False: the mixer has no
    key and value projections and reads the cache of the schedule entry it is pointed at; default True),
    ``cache_window`` (how many positions back the keys are kept, when that is not the mixer's own ``window`` or
    ``chunk``: the widest reach among this mixer and the mixers that read its cache), ``out_scale``.  Scores, weights
    and the weighted sum are float32 in every dtype."""

    def __init__(self, spec: PartSpec, position: Optional[PositionEncoding] = None):
        if position is None:
            from .recurrent import position_part
            position = position_part(spec.params)
        super().__init__(spec, position)
        p = spec.params
        self.hidden, self.nh, self.g, self.hs = int(p["hidden_size"]), int(p["num_heads"]), int(p["num_kv_heads"]), int(p["head_dim"])
        self.vd = int(p["v_head_dim"]) if p.get("v_head_dim") is not None else self.hs
        self.bias = bool(p.get("bias", False))
        self.norm_eps = float(p["qk_norm_eps"]) if p.get("qk_norm_eps") is not None else None
        self.scale = float(p["scale"]) if p.get("scale") is not None else 1.0 / math.sqrt(self.hs)
        self.softcap = float(p["softcap"]) if p.get("softcap") is not None else None
        self.learned_sink = p.get("sink") == "learned"
        self.sink = bool(p.get("sink", False))
        self.window = p.get("window")
        self.chunk = int(p["chunk"]) if p.get("chunk") is not None else None
        self.slopes_host = tuple(float(v) for v in p["distance_slopes"]) if p.get("distance_slopes") is not None else None
        self.norm_all = str(p.get("qk_norm_over", "head")) == "all"
        self.norm_weight = bool(p.get("qk_norm_weight", True))
        self.values_from_keys = bool(p.get("values_from_keys", False))
        db = p.get("distance_bias")
        self.distance_bias = (int(db["buckets"]), db["max"]) if db is not None else None
        self.pool = int(p["pool"]) if p.get("pool") is not None else None
        qt = p.get("q_temperature")
        self.q_temperature = (float(qt["coef"]), int(qt["every"])) if qt is not None else None
        self.gated = bool(p.get("gate", False))
        self.gate_per_head = p.get("gate") == "head"
        self.out_bias = bool(p.get("out_bias", False))
        self.own_kv = bool(p.get("own_kv", True))
        self.cache_window = p.get("cache_window", self.window if self.window is not None else self.chunk)
        if p.get("cache_window") is None and self.window is not None and self.chunk is not None:
            self.cache_window = min(self.window, self.chunk)
        self.out_scale = float(p.get("out_scale", 1.0))
        df = p.get("difference")
        self.difference = (float(df["offset"]), float(df["eps"])) if df is not None else None
        self.maps = 1 if df is None else 2
        self.combine: Optional[attn_ops.MapDifference] = None
        if df is not None and (self.sink or self.softcap is not None or self.chunk is not None or self.slopes_host is not None
                               or self.distance_bias is not None or self.pool is not None or self.gated or self.values_from_keys
                               or self.norm_all or not self.own_kv or self.out_scale != 1.0):
            raise ValueError("two maps per head go with a window, a norm per head and a rotation only")
        if self.slopes_host is not None and len(self.slopes_host) != self.nh:
            raise ValueError(f"{len(self.slopes_host)} distance slopes for {self.nh} heads")
        if self.chunk is not None and self.chunk <= 0 or self.q_temperature is not None and self.q_temperature[1] <= 0:
            raise ValueError("chunk and the query temperature's period must be positive")
        if self.distance_bias is not None:
            distance_bucket(0, *self.distance_bias)           # refuses what has no buckets
        if self.values_from_keys and (self.vd != self.hs or self.bias):
            raise ValueError("values that are the keys have the keys' head size and no bias of their own")
        if self.pool is not None:
            if self.pool <= 0 or self.window is None or self.chunk is not None or not self.own_kv:
                raise ValueError("pooled blocks need a window, a block size and keys of the mixer's own")
            # a block's mean is taken when its last token arrives: its tokens must be kept until then
            self.cache_window = max(self.cache_window, self.pool)
        if self.nh % self.g:
            raise ValueError(f"num_heads {self.nh} is not a multiple of num_kv_heads {self.g}")
        if max(self.hs, self.vd) > 256:
            raise ValueError(f"head sizes {self.hs}, {self.vd} are not supported (at most 256)")
        self.hidden_width = self.nh * self.vd
        self.shares_projections = not self.out_bias
        self.w_in: Optional[torch.Tensor] = None
        self.w_out: Optional[torch.Tensor] = None
        self.rel: Optional[torch.Tensor] = None
        self.biases = (None, None, None)
        self.q_norm = self.k_norm = None
        self.sink_logits = self.slopes = self.o_bias = None
        self.spans = {}

    def param_specs(self) -> Dict[str, ParamSpec]:
        qd, kd = self._query_rows(), self._key_rows()
        specs = {"q_proj": ParamSpec((qd, self.hidden)), "o_proj": ParamSpec((self.hidden, self.nh * self.vd))}
        if self.own_kv:
            specs["k_proj"] = ParamSpec((kd, self.hidden))
            if not self.values_from_keys:
                specs["v_proj"] = ParamSpec((self.g * self.vd, self.hidden))
        if self.bias:
            specs["q_bias"] = ParamSpec((qd,), init="zeros")
            if self.own_kv:
                specs.update({"k_bias": ParamSpec((kd,), init="zeros"), "v_bias": ParamSpec((self.g * self.vd,), init="zeros")})
        if self.norm_eps is not None and self.norm_weight:
            specs["q_norm"] = ParamSpec((self.nh * self.hs if self.norm_all else self.hs,), init="ones", keep_float32=True)
            if self.own_kv:
                specs["k_norm"] = ParamSpec((self.g * self.hs if self.norm_all else self.hs,), init="ones", keep_float32=True)
        if self.distance_bias is not None:
            specs["rel"] = ParamSpec((self.distance_bias[0], self.nh), init="zeros", keep_float32=True)
        if self.learned_sink:
            specs["sink"] = ParamSpec((self.nh,), init="zeros", keep_float32=True)
        if self.gated:
            specs["g_proj"] = ParamSpec((self.nh if self.gate_per_head else self.nh * self.vd, self.hidden))
        if self.out_bias:
            specs["o_bias"] = ParamSpec((self.hidden,), init="zeros", keep_float32=True)
        if self.difference is not None:
            specs.update({n: ParamSpec((self.hs,), keep_float32=True) for n in ("lq1", "lk1", "lq2", "lk2")})
        return specs

    def _query_rows(self) -> int:
        return self.nh * self.maps * self.hs

    def _key_rows(self) -> int:
        return self.g * self.maps * self.hs

    def load(self, t: Dict[str, torch.Tensor]) -> None:
        # the input matrices stacked, each block of the product's columns on a 16-byte boundary
        names = ["q_proj"] + (["k_proj"] if self.own_kv else []) + (["v_proj"] if "v_proj" in t else []) \
            + (["g_proj"] if self.gated else [])
        plain = not self.gated and self.own_kv and not self.values_from_keys
        if plain:
            self.w_in = torch.cat([t[n] for n in names], dim=0).contiguous()
            qd, kd = self._query_rows(), self._key_rows()
            spans = [(0, qd), (qd, qd + kd), (qd + kd, qd + kd + self.g * self.vd)]
        else:
            from .base import stack_rows
            self.w_in, spans = stack_rows([t[n] for n in names])
        self.spans = dict(zip(names, spans))
        self.w_out = t["o_proj"].contiguous()
        if self.bias:
            self.biases = tuple(t[n].to(self.w_in.dtype).contiguous() if n in t else None for n in ("q_bias", "k_bias", "v_bias"))
        if self.norm_eps is not None:
            sizes = (self.nh * self.hs, self.g * self.hs) if self.norm_all else (self.hs, self.hs)
            unit = [torch.ones(n, dtype=torch.float32, device=self.w_in.device) for n in sizes] if not self.norm_weight else None
            self.q_norm = unit[0] if unit else t["q_norm"].contiguous()
            self.k_norm = (unit[1] if unit else t["k_norm"].contiguous()) if self.own_kv else None
        if self.distance_bias is not None:
            # the table by distance, up to the window or to where every further distance shares the last number
            reach = distance_reach(*self.distance_bias)
            length = min(reach, self.window) if self.window is not None else reach
            index = torch.tensor([distance_bucket(n, *self.distance_bias) for n in range(length)], device=self.w_in.device)
            self.rel = t["rel"].float()[index].t().contiguous()
        if self.learned_sink:
            self.sink_logits = t["sink"].float().contiguous()
        if self.slopes_host is not None:
            self.slopes = torch.tensor(self.slopes_host, dtype=torch.float32, device=self.w_in.device)
        if self.out_bias:
            self.o_bias = t["o_bias"].float().contiguous()
        if self.difference is not None:
            dot = lambda a, b: float((t[a].double() * t[b].double()).sum())
            offset, eps = self.difference
            self.combine = attn_ops.MapDifference(math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + offset, eps)

    def in_weight(self) -> torch.Tensor:
        return self.w_in

    def out_weight(self) -> torch.Tensor:
        return self.w_out

    def release_projections(self) -> None:
        if self.out_bias:
            raise ValueError("an arrangement that adds several output products into one cannot carry this mixer's output bias")
        self.w_in = self.w_out = None

    def cache_request(self):
        vd = None if self.vd == self.hs else self.vd
        if self.difference is not None:
            return PagedKV(self.g, self.maps * self.hs, self.cache_window, v_head_dim=self.vd)
        tokens = PagedKV(self.g, self.hs, self.cache_window, v_head_dim=vd)
        if self.pool is None:
            return tokens
        return {"tokens": tokens, "blocks": PagedKV(self.g, self.hs, None, v_head_dim=vd, pool=self.pool)}

    def _tensor_core_form(self, dtype: torch.dtype) -> bool:
        """bfloat16 steps with head sizes the kernel is built for go to the tensor cores (scores and the sum of weights
        in float32, the weights against V in two bfloat16 halves); float32 steps and other shapes go to the exact
        kernel."""
        if dtype != torch.bfloat16:
            return False
        if self.difference is not None:
            return attn_ops.mma_maps_supports(self.hs, self.vd)
        plain = self.vd == self.hs and self.distance_bias is None and self.pool is None and attn_ops.mma_supports(self.hs)
        return plain or attn_ops.mma_extended_supports(self.hs, self.vd)

    def _launch_shape(self, host):
        """(longest portion, key splits): a step in which a request's rows fill at most one tile of 16 (single
        tokens of up to 16 heads per group) may divide each request's keys among blocks."""
        rows = host.max_q_len * (self.nh // self.g)
        blocks = self.g * (2 if self.difference is not None and rows > 8 else 1)      # two maps: eight rows of each a block
        return host.max_q_len, (attn_ops.decode_splits(len(host.slots), blocks) if rows <= 16 else 1)

    def capture_key(self, host):
        # the exact kernel launches the same for every step; the tensor-core one by the longest portion
        return ("general_attention",) + self._launch_shape(host)

    def keys_seen(self, position: int) -> int:
        """How many keys the query at ``position`` sees."""
        lo = max(0, position - self.window + 1) if self.window else 0
        if self.chunk:
            lo = max(lo, position // self.chunk * self.chunk)
        return position - lo + 1

    def blocks_seen(self, position: int) -> int:
        """How many pooled blocks the query at ``position`` sees."""
        return max(0, position - self.window + 1) // self.pool if self.pool else 0

    def mixing_flops(self, q_len: int, ctx_before: int) -> float:
        keys = sum(self.keys_seen(ctx_before + t) + self.blocks_seen(ctx_before + t) for t in range(q_len)) if self.window or self.chunk \
            else q_len * ctx_before + q_len * (q_len + 1) / 2
        return 2.0 * self.nh * self.maps * (self.hs + self.vd) * keys

    def mix(self, z: torch.Tensor, ctx, cache, y: torch.Tensor) -> None:
        if self.position is None:
            freq, interleaved, magnitude = None, False, 1.0
        else:
            interleaved = bool(getattr(self.position, "interleaved", False))
            magnitude = float(getattr(self.position, "magnitude", 1.0))
            freq = self.position.frequencies(self.position.head_dim, z.device)
        blocks = None
        if self.pool is not None:
            cache, blocks = cache["tokens"], cache["blocks"]
            blocks = attn_ops.PooledBlocks(self.pool, blocks.k, blocks.v, ctx.block_tables[blocks.group])
        table = ctx.block_tables[cache.group]
        if self.own_kv != cache.writable:
            raise ValueError("a mixer with key and value projections writes its own cache; one without reads another's")
        q_at = self.spans["q_proj"][0]
        k_at = self.spans["k_proj"][0] if self.own_kv else q_at
        v_at = self.spans["v_proj"][0] if "v_proj" in self.spans else k_at
        pooling = {} if blocks is None else dict(pool=blocks.size, pooled_k=blocks.k, pooled_v=blocks.v, pooled_table=blocks.table,
                                                 single_tokens=ctx.host.max_q_len == 1)
        q = qkv_prepare(z, (q_at, k_at, v_at), self.nh * self.maps, self.g, self.hs, self.vd, ctx.positions, ctx.req_of_token,
                        out_dtype=z.dtype, biases=self.biases, q_norm=self.q_norm, k_norm=self.k_norm,
                        norm_eps=self.norm_eps or 0.0, inv_freq=freq, k_pool=cache.k, v_pool=cache.v, block_table=table,
                        store=cache.writable, bad_flag=ctx.error_flag, interleaved=interleaved,
                        q_temperature=self.q_temperature, rot_scale=magnitude, norm_all=self.norm_all,
                        maps=self.maps, **pooling)
        gate = None
        if self.gated:
            a, b = self.spans["g_proj"]
            gate = z[:, a:b]
        extras = dict(chunk=self.chunk, sink_logits=self.sink_logits, slopes=self.slopes, gate=gate, rel=self.rel, pool=blocks,
                      v_head_dim=self.vd)
        scale_out = self.out_scale if self.difference is None else 1.0 - self.difference[0]
        if self._tensor_core_form(z.dtype):
            longest, splits = self._launch_shape(ctx.host)
            direct = y.data_ptr() % 16 == 0 and y.stride(0) % 2 == 0
            out = attn_ops.paged_attention_mma(q, cache.k, cache.v, ctx.positions, ctx.q_start, ctx.req_of_token, table, longest,
                                               self.nh, self.g, self.hs, scale=self.scale, window=self.window, n_splits=splits,
                                               out=y if direct else None, softcap=self.softcap, sink=self.sink,
                                               out_scale=scale_out, exact_weights=True, difference=self.combine, **extras)
            if not direct:
                y.copy_(out)
            return
        attn_ops.paged_attention_generic(q, cache.k, cache.v, ctx.positions, ctx.req_of_token, table, self.nh, self.g, self.hs,
                                         scale=self.scale, window=self.window, out=y,
                                         softcap=self.softcap, sink=self.sink, out_scale=scale_out, difference=self.combine, **extras)

    def forward(self, x: torch.Tensor, ctx, cache: PagedKVCache):
        out = self.project_and_mix(x, ctx, cache)
        return NormedSum(out, bias=self.o_bias) if self.out_bias else out


register_part("mixer", "paged_attention", PagedAttention)
register_part("mixer", "general_attention", GeneralAttention)

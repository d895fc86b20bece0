"""The attention mixer: grouped-query causal attention over the paged cache."""
from __future__ import annotations

import torch

from ..cache import CacheNeed, StateNeed
from ..config import PartSpec
from ..ops import kernels
from ..ops.linear import Linear
from .registry import POSITION_ENCODINGS, build_part, register_mixer


@register_mixer("attention")
class AttentionMixer:
    """q, k, v = W_qkv xn; position encoding on q and k; k, v stored in the request's pages;
    causal softmax(q k^T * scale) v per head with query head h reading key/value head
    h // (H / Hkv); x += W_o out (src/model/transformer.cpp:389-434).

    Params: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``scale`` (multiplied
    after the dot product), ``window`` (None = all keys) and ``position`` (a PartSpec).
    Weights: ``w_qkv`` [(H+2Hkv)*hd, hidden] and ``w_o`` [hidden, H*hd].

    Options (each absent by default; any of them takes the mixer off the fused [q; k; v] product with
    rotation in its epilogue and onto the 32-bit projection followed by the norm+rotation+store kernel):
    ``values`` = "keys": the model has no value projection; the value rows written to the pages are the key
    projection's raw output, taken ahead of the per-head norm and the rotation (``w_qkv`` then has no value rows). ``qk_norm_eps``: queries and keys are
    normalised per head to unit RMS and multiplied by ``q_norm`` / ``k_norm`` [hd] (shared by the heads)
    before the rotation. ``sink``: the softmax's denominator has one more term, exp(0). ``head_gate``:
    ``w_qkv`` ends with H more rows, and head h's output is multiplied by the sigmoid of its row's product
    with the input. ``out_scale``: a constant on the mixer's output (applied before the output projection).

    Further options, which run the row-form attention kernel (32-bit arithmetic over shared key tiles):
    ``value_dim``: value heads of a width of their own (``w_qkv`` then has Hkv * value_dim value rows, ``w_o``
    H * value_dim columns, and the values have pages of their own). ``qk_norm_weights`` False: the unit-RMS norm of
    queries and keys has no weights. ``distance_slopes`` [H]: slope_h * (i - j) is taken off the score of key j for the
    query at i. ``chunk``: position i sees j <= i only inside its own block of ``chunk`` positions counted from 0
    (pages of earlier blocks are given back). ``sink`` = "learned": the term added to the softmax's denominator is
    exp(``sink``_h) with a weight per head (``sink`` [H]). ``softcap`` c: the scaled score s becomes c tanh(s / c).

    ``qk_norm_wide`` (with ``qk_norm_eps``): the norm runs over the whole query projection at once (all heads' values
    together, ``q_norm`` [H * hd]) and over the whole key projection (``k_norm`` [Hkv * hd]) instead of head by head.
    ``conv_taps`` n: every channel of the [q; k; v] projection passes a causal convolution over the request's last n
    tokens before anything else (``conv`` [channels, n], column n-1 weighs the newest token; no bias, no activation;
    nothing before the first token; one tap is a factor per channel); the request's last n-1 projected rows are state, kept
    in its state slot from ``state_offset`` on.

    ``bias``: q, k and v have biases, added in 32-bit to the projection before the norm and the rotation (``b_qkv`` [(H + Hkv) hd +
    Hkv vd]). ``output_gate``: ``w_qkv`` ends with H vd more rows, and every value of the heads' outputs is multiplied by the
    sigmoid of its row's product with the input (in the attention kernels' last step).

    ``maps`` = 2 (with ``map_weight`` and ``map_factor``): every head has two score maps over the same values. ``num_heads`` and
    ``num_kv_heads`` count heads, ``head_dim`` is the width of one map; a head's queries and keys are [map 1, map 2] in
    ``w_qkv`` (2 H hd query rows, 2 Hkv hd key rows), each map brought to unit RMS and weighted on its own (``qk_norm_eps``,
    ``q_norm`` and ``k_norm`` [hd]). With a1, a2 the maps' attention outputs and w = exp(sum lq1 lk1) - exp(sum lq2 lk2) +
    map_weight (weights ``lq1``, ``lk1``, ``lq2``, ``lk2`` [hd]), a head's output is map_factor * N(a1 - w a2), N to unit RMS over the
    value width (eps ``qk_norm_eps``). ``query_temperature`` (coef, every): the queries at position p are multiplied by
    1 + coef ln(floor((p + 1) / every) + 1). The cache holds [map 1, map 2] in one key row per key head; to the attention
    kernels these are 2 H query heads ([map 1, 0] and [0, map 2]) over Hkv key heads of 2 hd, which share the rows they read.
    In bfloat16, rows of keys and values are widened with zeros to a width that the tensor-core kernels are built for where that
    at most doubles them; other sizes and the 32-bit path run the row-form kernel."""

    graph_safe = True      # launches depend only on the step's shape: decode steps may be captured in a CUDA graph


    def __init__(self, params, weights, build):
        self.hidden_size = int(params["hidden_size"])
        self.num_heads = int(params["num_heads"])
        self.num_kv_heads = int(params["num_kv_heads"])
        self.head_dim = int(params["head_dim"])
        self.scale = float(params["scale"])
        self.window = params.get("window")
        if self.num_heads % self.num_kv_heads:
            raise ValueError("attention: num_heads must be a multiple of num_kv_heads")
        self.maps = int(params.get("maps", 1))
        self.temperature = None
        if self.maps not in (1, 2):
            raise ValueError("attention: heads have one score map or two")
        if self.maps == 2:
            self._init_maps(params, weights, build)
        elif not kernels.attention_supported(self.head_dim):
            raise ValueError(f"attention: head size {self.head_dim} is not supported by the attention kernels "
                             f"(up to 256)")
        pos_spec = params.get("position") or PartSpec("none", {})
        self.position = build_part(POSITION_ENCODINGS, "position encoding", pos_spec, {}, build)
        self.values_are_keys = params.get("values", "projected") == "keys"
        if params.get("values", "projected") not in ("projected", "keys"):
            raise ValueError(f"attention: unknown source of values '{params.get('values')}'")
        self.qk_norm_eps = params.get("qk_norm_eps")
        if self.maps == 1:
            self.value_dim = int(params.get("value_dim") or self.head_dim)
        self.chunk = params.get("chunk")
        self.learned_sink = params.get("sink") == "learned"
        self.softcap = float(params["softcap"]) if params.get("softcap") else None
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError("attention: the soft cap of the scores must be positive")
        self.wide_norm = bool(params.get("qk_norm_wide", False))
        self.conv_taps = int(params["conv_taps"]) if params.get("conv_taps") else None
        self.state_offset = 0
        slopes = params.get("distance_slopes")
        if slopes is not None and len(slopes) != self.num_heads:
            raise ValueError("attention: distance_slopes needs one slope per head")
        self.slopes = None if slopes is None else torch.tensor([float(v) for v in slopes], dtype=torch.float32, device=build.device)
        # these options are served by the row-form kernel only
        self.row_form = (self.value_dim != self.head_dim or self.chunk is not None or self.learned_sink or
                         self.slopes is not None or self.softcap is not None)
        if self.maps == 2:        # two maps: the row-form kernel wherever the tensor-core kernels are not built for the sizes
            self.row_form = self.row_form or build.compute_dtype is not torch.bfloat16 or \
                not kernels.attention_fast_supported(self.head_dim, self.num_heads, self.num_kv_heads)
        self.sink = bool(params.get("sink", False))
        self.head_gate = bool(params.get("head_gate", False))
        self.output_gate = bool(params.get("output_gate", False))
        if self.output_gate and (self.head_gate or params.get("conv_taps") or self.maps == 2):
            raise ValueError("attention: an output gate cannot be combined with a head gate, a convolution or two score maps")
        if params.get("bias") and (self.values_are_keys or params.get("conv_taps") or self.maps == 2):
            raise ValueError("attention: biases cannot be combined with values taken from the keys, a convolution or two score maps")
        self.out_scale = float(params.get("out_scale", 1.0))
        on_device = getattr(self.position, "freq", None) is not None
        self.extended = (self.output_gate or bool(params.get("bias")) or self.values_are_keys or self.qk_norm_eps is not None or self.sink or self.head_gate
                         or self.out_scale != 1.0 or on_device or self.row_form or self.conv_taps is not None)
        if self.row_form:
            if self.head_gate or self.out_scale != 1.0 or self.values_are_keys:
                raise ValueError("attention: a gate, an output factor or values taken from the keys cannot be combined with "
                                 "value_dim, chunk, distance_slopes, a soft cap or a learned sink")
            if not kernels.attention_rows_supported(self.head_dim, self.value_dim):
                raise ValueError(f"attention: head size {self.head_dim} with value size {self.value_dim} is not supported")
        if getattr(self.position, "amplitude", 1.0) != 1.0:
            raise ValueError("attention: a rotation whose cos and sin are scaled is not served by this mixer")
        self.sink_weight = None
        if self.learned_sink:
            if tuple(weights["sink"].shape) != (self.num_heads,):
                raise ValueError(f"attention: sink has shape {tuple(weights['sink'].shape)}, expected ({self.num_heads},)")
            self.sink_weight = weights["sink"].to(device=build.device, dtype=torch.float32).contiguous()
        elif self.row_form and self.sink:
            self.sink_weight = torch.zeros(self.num_heads, dtype=torch.float32, device=build.device)      # exp(0) = 1
        if self.extended and getattr(self.position, "cos", None) is not None:
            raise ValueError("attention: with these options the rotation's angles are computed on the device "
                             "(position encoding 'rope_on_device' or 'none')")
        # soft-capped scores alone (equal key and value sizes, nothing else of the row form): prompt portions may run on the
        # tcgen05 kernel and single tokens on the decode kernel, which have the cap
        self.cap_only = (self.softcap is not None and self.value_dim == self.head_dim and self.chunk is None and self.slopes is None
                         and not self.learned_sink and not params.get("sink") and build.compute_dtype is torch.bfloat16)
        self.q_norm = self.k_norm = None
        if self.maps == 2:
            self.q_norm, self.k_norm = (_vector_of(weights, n, self.map_dim, build) for n in ("q_norm", "k_norm"))
        elif self.qk_norm_eps is not None and not params.get("qk_norm_weights", True):
            self.q_norm = self.k_norm = torch.ones(self.head_dim, dtype=torch.float32, device=build.device)
        elif self.qk_norm_eps is not None:
            for name, heads in (("q_norm", self.num_heads), ("k_norm", self.num_kv_heads)):
                n = heads * self.head_dim if self.wide_norm else self.head_dim
                if tuple(weights[name].shape) != (n,):
                    raise ValueError(f"attention: {name} has shape {tuple(weights[name].shape)}, expected ({n},)")
                setattr(self, name, weights[name].to(device=build.device, dtype=torch.float32).contiguous())
        if self.wide_norm and (self.qk_norm_eps is None or not params.get("qk_norm_weights", True)):
            raise ValueError("attention: qk_norm_wide needs qk_norm_eps and weights")
        if self.maps == 2:
            qkv_rows = 2 * (self.map_heads + self.num_kv_heads) * self.map_dim + self.num_kv_heads * self.map_value_dim
            out_columns = self.map_heads * self.map_value_dim
        else:
            qkv_rows = (self.num_heads + self.num_kv_heads) * self.head_dim + \
                (0 if self.values_are_keys else self.num_kv_heads * self.value_dim) + (self.num_heads if self.head_gate else 0) + \
                (self.num_heads * self.value_dim if self.output_gate else 0)
            out_columns = self.num_heads * self.value_dim
        if tuple(weights["w_qkv"].shape) != (qkv_rows, self.hidden_size):
            raise ValueError(f"attention: w_qkv has shape {tuple(weights['w_qkv'].shape)}, expected "
                             f"({qkv_rows}, {self.hidden_size})")
        if tuple(weights["w_o"].shape) != (self.hidden_size, out_columns):
            raise ValueError(f"attention: w_o has shape {tuple(weights['w_o'].shape)}")
        self.bias = None
        if params.get("bias"):          # zeros behind: a gate's columns have none
            n = (self.num_heads + self.num_kv_heads) * self.head_dim + self.num_kv_heads * self.value_dim
            self.bias = torch.zeros(qkv_rows, dtype=torch.float32, device=build.device)
            self.bias[:n] = _vector_of(weights, "b_qkv", n, build)
        self.conv = None
        if self.conv_taps is not None:
            if self.head_gate or self.values_are_keys:
                raise ValueError("attention: a convolution of the projections cannot be combined with a head gate or values taken from the keys")
            if not (self.conv_taps <= 17):
                raise ValueError(f"attention: {self.conv_taps} convolution taps are not supported (1 to 17)")
            if tuple(weights["conv"].shape) != (qkv_rows, self.conv_taps):
                raise ValueError(f"attention: conv has shape {tuple(weights['conv'].shape)}, expected ({qkv_rows}, {self.conv_taps})")
            self.conv = weights["conv"].to(device=build.device, dtype=torch.float32).contiguous()
            self.conv_channels = qkv_rows
        self.w_qkv = Linear(weights["w_qkv"], build.compute_dtype, build.device, tiles=build.weight_tiles)
        self.w_o = Linear(weights["w_o"], build.compute_dtype, build.device, tiles=build.weight_tiles)
        self.dtype = build.compute_dtype
        # bfloat16 with a head size the tensor-core kernels are built for; else the general kernel
        self.fast = self.dtype is torch.bfloat16 and not self.row_form and kernels.attention_fast_supported(
            self.head_dim, self.num_heads, self.num_kv_heads)
        self._prefill_rows = {}
        self.cap_fast = self.cap_only and kernels.attention_fast_supported(self.head_dim, self.num_heads, self.num_kv_heads)
        if self.fast or self.cap_fast:
            self.chunk_keys = kernels.attention_chunk_keys()
            self.max_chunks = (build.max_position + self.chunk_keys - 1) // self.chunk_keys

    def _init_maps(self, params, weights, build) -> None:
        """Heads of two score maps: from here on ``num_heads`` and ``head_dim`` are what the attention kernels see."""
        for option in ("window", "chunk", "sink", "softcap", "head_gate", "distance_slopes", "conv_taps", "qk_norm_wide"):
            if params.get(option):
                raise ValueError(f"attention: '{option}' cannot be combined with two score maps")
        if params.get("values", "projected") != "projected" or params.get("out_scale", 1.0) != 1.0 or \
                (params.get("position") is not None and params["position"].kind != "none"):
            raise ValueError("attention: two score maps take projected values, no output factor and no rotation")
        if params.get("qk_norm_eps") is None or not params.get("qk_norm_weights", True):
            raise ValueError("attention: two score maps need qk_norm_eps and weights")
        self.map_heads, self.map_dim = self.num_heads, self.head_dim
        vd = self.map_value_dim = int(params.get("value_dim") or self.map_dim)
        self.num_heads, self.head_dim, self.value_dim = 2 * self.num_heads, 2 * self.head_dim, vd
        if build.compute_dtype is torch.bfloat16:
            widest = max(self.head_dim, vd)
            width = next((w for w in (16, 32, 64, 128) if w >= widest), None)
            if width and 2 * width <= 2 * (self.head_dim + vd) and \
                    kernels.attention_fast_supported(width, self.num_heads, self.num_kv_heads):
                self.head_dim = self.value_dim = width
        if not kernels.attention_rows_supported(self.head_dim, vd) or not kernels.maps_combine_supported(vd):
            raise ValueError(f"attention: two maps of size {self.map_dim} with value size {vd} are not supported")
        lq1, lk1, lq2, lk2 = (_vector_of(weights, n, self.map_dim, build).double() for n in ("lq1", "lk1", "lq2", "lk2"))
        self.map_weight = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + float(params["map_weight"])
        self.map_factor = float(params["map_factor"])
        if params.get("query_temperature"):
            coef, every = (float(v) for v in params["query_temperature"])
            if not every > 0:
                raise ValueError("attention: the query temperature's blocks must have a positive length")
            self.temperature = (coef, every)

    def prefill_on_tcgen05(self, page_size: int) -> bool:
        """Head sizes 64 and 128 with pages TMA can tile: prompt portions run on the tcgen05 kernel."""
        key = ("tc", page_size)
        if key not in self._prefill_rows:
            self._prefill_rows[key] = kernels.attention_prefill_tc_supported(self.head_dim, self.num_heads,
                                                                             self.num_kv_heads, page_size)
        return self._prefill_rows[key]

    def prefill_rows(self, page_size: int) -> int:
        """Query rows (tokens x heads of a group) per work item of the prefill kernel in use."""
        if page_size not in self._prefill_rows:
            self._prefill_rows[page_size] = 128 if self.prefill_on_tcgen05(page_size) else \
                kernels.attention_prefill_rows(page_size, self.head_dim)
        return self._prefill_rows[page_size]

    def cache_need(self):
        return CacheNeed(self.num_kv_heads, self.head_dim, self.window,
                         value_dim=None if self.value_dim == self.head_dim else self.value_dim, chunk=self.chunk)

    def state_need(self):
        if self.conv is None or self.conv_taps == 1:
            return None
        return StateNeed(((self.conv_taps - 1) * self.conv_channels,), "float32")

    def launch_key(self, ctx, run):
        key = self._launch_key(ctx, run)
        return key + (ctx.n_requests,) if self.conv is not None else key

    def _launch_key(self, ctx, run):
        """What the mixer's launches depend on besides the token count: whose cache it uses, and (tensor-core
        kernels) how many rows are single decoded tokens, how many tiles the prompt portions make and how many
        chunks the longest context of a single token has. Asking also places this step's work lists on the device."""
        if self.row_form:
            key = (run.cache_layer, run.writes_cache) + kernels.attention_rows_launch_key(
                ctx, self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, False, self.dtype)
            if self._cap_tiles_on_tcgen05(ctx):
                key += (ctx.attention_work(128 // (self.num_heads // self.num_kv_heads))[1].shape[0],)
            if self._cap_singles_on_decode(ctx):
                per_tile = kernels.attention_rows_tile_tokens(self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, False)
                key += ((ctx.attention_work(per_tile)[2] + self.chunk_keys - 1) // self.chunk_keys,)
            return key
        if not self._fast_now(ctx):
            return (run.cache_layer, run.writes_cache)
        rows, work, longest = ctx.attention_work(self.prefill_rows(ctx.page_size) // (self.num_heads // self.num_kv_heads))
        return (run.cache_layer, run.writes_cache, rows.numel(), work.shape[0],
                (longest + self.chunk_keys - 1) // self.chunk_keys)

    takes_then = True      # forward accepts ``then``

    def _cap_singles_on_decode(self, ctx) -> bool:
        return (self.cap_fast and hasattr(ctx, "attention_work") and kernels.attention_tma_pages(ctx.page_size)
                and kernels.attention_rows_tile_tokens(self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, False) > 0)

    def _cap_tiles_on_tcgen05(self, ctx) -> bool:
        return (self.cap_only and hasattr(ctx, "attention_work") and self.prefill_on_tcgen05(ctx.page_size)
                and kernels.attention_rows_tile_tokens(self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, False) > 0)

    def _fast_now(self, ctx) -> bool:
        """Whether this step's attention runs on the tensor-core kernels: bfloat16 with a head size they are built for;
        with a sink, a gate or an output factor also pages that their TMA-fed forms can tile."""
        return self.fast and (not self.extended or kernels.attention_tma_pages(ctx.page_size))

    def _attend(self, ctx, q, k_cache, v_cache, att, tables, **epilogue) -> None:
        """Attention of the step's rows: single decoded tokens split their context over many CTAs, portions of
        prompts run tile by tile (tensor cores); else the general kernel. ``epilogue``: sink, gate, gate_offset, gate_dims, out_scale."""
        H, Hkv, hd = self.num_heads, self.num_kv_heads, self.head_dim
        if not self._fast_now(ctx):
            kernels.attention_generic(q, k_cache, v_cache, att, ctx.row_req, ctx.positions, tables, H, Hkv, hd,
                                      ctx.page_size, self.scale, self.window, **epilogue)
            return
        rows, work, longest = ctx.attention_work(self.prefill_rows(ctx.page_size) // (H // Hkv))
        if rows.numel():
            n = rows.numel()
            part_o = ctx.scratch("att_part_o", (n, H * self.max_chunks * hd), torch.float32, capacity=ctx.max_requests)
            part_ml = ctx.scratch("att_part_ml", (n, H * self.max_chunks * 2), torch.float32, capacity=ctx.max_requests)
            n_chunks = (longest + self.chunk_keys - 1) // self.chunk_keys
            kernels.attention_decode(q, k_cache, v_cache, att, rows, ctx.row_req, ctx.positions, tables, H, Hkv, hd,
                                     ctx.page_size, self.scale, self.window, part_o, part_ml, self.max_chunks, n_chunks,
                                     **epilogue)
        if work.shape[0]:
            prefill = kernels.attention_prefill_tc if self.prefill_on_tcgen05(ctx.page_size) else kernels.attention_prefill
            prefill(q, k_cache, v_cache, att, work, ctx.positions, tables, H, Hkv, hd, ctx.page_size, self.scale,
                    self.window, **epilogue)

    def forward(self, ctx, run, xn: torch.Tensor, x: torch.Tensor, then=None) -> None:
        """``xn``: normalised input [T, hidden] in the compute dtype; ``x``: the 32-bit residual
        stream, to which the mixer's output is added. ``run`` names whose cache to use. ``then``: the Linear
        of the large product that follows this mixer (the feed-forward's first), for the last product here to
        ask the start of its weights into L2."""
        T = xn.shape[0]
        H, Hkv, hd = self.num_heads, self.num_kv_heads, self.head_dim
        k_cache, v_cache = ctx.pages(run.cache_layer)
        tables = ctx.block_tables(run.cache_layer)
        q = ctx.scratch("q", (T, H * hd), self.dtype)
        if self.extended:
            self._forward_extended(ctx, run, xn, x, q, k_cache, v_cache, tables, then)
            return
        if self.dtype is torch.bfloat16 and kernels.gemm_rope_store_supported(
                T, self.hidden_size, H, Hkv, hd, self.position.cos, self.position.interleaved):
            # rotation and page store in the epilogue of the product
            kernels.gemm_rope_store(xn, self.w_qkv.weight, ctx.positions, ctx.row_req, tables, self.position.cos,
                                    self.position.sin, self.position.interleaved, q, k_cache, v_cache, H, Hkv, hd,
                                    ctx.page_size, write_kv=run.writes_cache, w_tiles=self.w_qkv.weight_tiles)
        else:
            qkv = ctx.scratch("qkv", (T, (H + 2 * Hkv) * hd), torch.float32)
            self.w_qkv.forward(xn, qkv)
            kernels.rope_store(qkv, ctx.positions, ctx.row_req, tables, self.position.cos, self.position.sin,
                               self.position.interleaved, q, k_cache, v_cache, H, Hkv, hd, ctx.page_size,
                               write_kv=run.writes_cache)
        att = ctx.scratch("att", (T, H * hd), self.dtype)
        self._attend(ctx, q, k_cache, v_cache, att, tables)
        self.w_o.forward(att, x, accumulate=True, then=then)

    def _forward_extended(self, ctx, run, xn, x, q, k_cache, v_cache, tables, then) -> None:
        """The mixer with options: projections to 32-bit, then per head norm, rotation and page store, attention
        with sink and gate in its epilogue, and the output projection."""
        T = xn.shape[0]
        H, Hkv, hd = self.num_heads, self.num_kv_heads, self.head_dim
        proj = ctx.scratch("att_proj", (T, self.w_qkv.out_features), torch.float32)
        self.w_qkv.forward(xn, proj)
        if self.conv is not None:
            mixed = ctx.scratch("att_proj_conv", (T, self.conv_channels), torch.float32)
            state = ctx.state(run.cache_layer) if self.conv_taps > 1 else mixed      # one tap reaches no earlier token: no state is touched
            kernels.causal_conv(proj, 0, self.conv, None, state, self.state_offset if self.conv_taps > 1 else 0, ctx.row_req,
                                ctx.seg_start, ctx.seg_len, ctx.state_slots, mixed, activate=False)
            proj = mixed
        if self.maps == 2:
            k_off = 2 * self.map_heads * self.map_dim
            kernels.maps_norm_store(proj, 0, k_off, k_off + 2 * Hkv * self.map_dim, self.q_norm, self.k_norm, self.qk_norm_eps,
                                    self.temperature, ctx.positions, ctx.row_req, tables, q, k_cache, v_cache, self.map_heads, Hkv,
                                    self.map_dim, self.map_value_dim, ctx.page_size, write_kv=run.writes_cache)
            self._attend_maps(ctx, q, k_cache, v_cache, tables, x, then)
            return
        k_off = H * hd
        v_off = k_off if self.values_are_keys else k_off + Hkv * hd
        gate_off = v_off + Hkv * self.value_dim
        kernels.norm_rope_store(proj, 0, k_off, v_off, self.q_norm, self.k_norm, self.qk_norm_eps or 0.0,
                                getattr(self.position, "freq", None), self.position.interleaved, ctx.positions,
                                ctx.row_req, tables, q, k_cache, v_cache, H, Hkv, hd, ctx.page_size,
                                write_kv=run.writes_cache, value_dim=self.value_dim, wide_norm=self.wide_norm, bias=self.bias)
        # (a gate per head, or one per value laid out as the heads' outputs)
        gate = {"gate": proj if self.head_gate or self.output_gate else None, "gate_offset": gate_off}
        gate_dims = self.value_dim if self.output_gate else 0
        if self.row_form:
            att = ctx.scratch("att", (T, H * self.value_dim), self.dtype)
            tiles_on = None
            if self._cap_tiles_on_tcgen05(ctx):
                tiles_on = (128 // (H // Hkv), lambda work: kernels.attention_prefill_tc(
                    q, k_cache, v_cache, att, work, ctx.positions, tables, H, Hkv, hd, ctx.page_size, self.scale, self.window,
                    softcap=self.softcap, gate_dims=gate_dims, **gate))
            singles_on = None
            if self._cap_singles_on_decode(ctx):
                def singles_on(rows, longest):
                    n = rows.numel()
                    part_o = ctx.scratch("att_part_o", (n, H * self.max_chunks * hd), torch.float32, capacity=ctx.max_requests)
                    part_ml = ctx.scratch("att_part_ml", (n, H * self.max_chunks * 2), torch.float32, capacity=ctx.max_requests)
                    kernels.attention_decode(q, k_cache, v_cache, att, rows, ctx.row_req, ctx.positions, tables, H, Hkv, hd,
                                             ctx.page_size, self.scale, self.window, part_o, part_ml, self.max_chunks,
                                             (longest + self.chunk_keys - 1) // self.chunk_keys, softcap=self.softcap,
                                             gate_dims=gate_dims, **gate)
            kernels.attention_rows_of_step(ctx, q, k_cache, v_cache, att, tables, H, Hkv, hd, self.value_dim, self.scale,
                                           self.window, self.chunk, self.slopes, self.sink_weight, softcap=self.softcap,
                                           tiles_on=tiles_on, singles_on=singles_on, **gate)
            self.w_o.forward(att, x, accumulate=True, then=then)
            return
        att = ctx.scratch("att", (T, H * hd), self.dtype)
        self._attend(ctx, q, k_cache, v_cache, att, tables, sink=self.sink, out_scale=self.out_scale, gate_dims=gate_dims, **gate)
        self.w_o.forward(att, x, accumulate=True, then=then)

    def _attend_maps(self, ctx, q, k_cache, v_cache, tables, x, then) -> None:
        """Both maps of every head in one attention call, then their difference and the output projection."""
        T, H, vd = q.shape[0], self.num_heads, self.value_dim
        if self.row_form:
            both = ctx.scratch("att_maps", (T, H * vd), torch.float32)
            kernels.attention_rows_of_step(ctx, q, k_cache, v_cache, both, tables, H, self.num_kv_heads, self.head_dim, vd, self.scale,
                                           None, None, None, None)
        else:
            both = ctx.scratch("att_maps", (T, H * vd), self.dtype)
            self._attend(ctx, q, k_cache, v_cache, both, tables)
        att = ctx.scratch("att", (T, self.map_heads * self.map_value_dim), self.dtype)
        kernels.maps_combine(both, att, self.map_weight, self.qk_norm_eps, self.map_factor, self.map_heads)
        self.w_o.forward(att, x, accumulate=True, then=then)


def _vector_of(weights, name: str, n: int, build) -> torch.Tensor:
    w = weights[name]
    if tuple(w.shape) != (n,):
        raise ValueError(f"attention: {name} has shape {tuple(w.shape)}, expected ({n},)")
    return w.to(device=build.device, dtype=torch.float32).contiguous()

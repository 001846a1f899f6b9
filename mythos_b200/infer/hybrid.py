"""Inference engine of layer-list models (:mod:`mythos_b200.models.hybrid_config`).

``HybridEngine`` is an :class:`InferenceEngine`: generation, the step-wise API, sampling, the page
allocator and the CUDA-graph decode loop are the base class's. It brings its own pass over the layers
and, beside the attention layers' pages, a slot of recurrent state per sequence.

A pass takes a ragged batch (new tokens of several sequences, packed; prompts, portions of prompts and
single decoded tokens in any mix). The residual stream is fp32; a sublayer reads its normalised copy in
the engine's activation type. All projections of a mixer that read the same input are one GEMM. Per
gated-linear-attention layer: projections -> decay GEMM -> recurrence -> head norm * gate -> output
GEMM -> (post-norm + residual + next pre-norm). A parallel layer runs a recurrence and paged attention side by
side: with norms of their own their outputs are averaged inside that last kernel, with constant scales both write
into one row and share one output GEMM.

Attention: one kernel turns the projection into queries and cached keys and values (bias, head norm, rotation,
query temperature), one attends (window, sink, output gate). Heads are stored padded to a multiple of 8 columns. A
layer that shares another's keys and values only forms queries. Selective scan: convolution -> GEMM to step sizes
and input / read-out maps -> GEMM to the channels' step sizes -> scan with its output gate.

Latent attention caches one row per token (latent | rotated key part) that all heads share. Tokens of
sequences that bring few of them at once (decoding, short portions) attend in the latent's space: queries go
through W_uk, the result through W_uv. Longer portions expand the latents of their sequence to keys and
values once per pass (with a window those of its reach) and run the tensor-core prompt attention. A batch with both
runs both. The order of rotated columns is free, so halves are stored as neighbouring pairs. Routed experts:
router GEMM -> selection and row segments -> row gather -> two grouped GEMMs -> (weighted sum + shared expert +
norm + residual).

Parallel designs: mixer and feed-forward write side by side into one row and share one output GEMM; one kernel adds it
to the stream and normalises, and for single tokens also runs the convolution in front of the next mixer (its last
inputs are a state of every layer). Longer portions run that convolution as a kernel of its own.

``dtype``: "bfloat16" (matrix products and activations in bf16 with 32-bit accumulation; residual,
norms, decays, states and scores in 32-bit) or "float32" (everything in 32-bit).
"""
from __future__ import annotations

import math

import torch

from ..models.hybrid_config import (AttentionMixer, HybridConfig, LatentAttentionMixer, MoeFF, ParallelMixer, RecurrentMixer,
                                    SelectiveMixer)
from ..ops import native
from .engine import InferenceEngine
from .kv_paged import PagedKVCache, RecurrentStatePool

DTYPES = {"bfloat16": torch.bfloat16, "bf16": torch.bfloat16, "float32": torch.float32, "fp32": torch.float32}


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _pad_heads(w: torch.Tensor, heads: int) -> torch.Tensor:
    """Rows (or values) of every head padded with zeros to a multiple of 8."""
    width = w.shape[0] // heads
    out = w.new_zeros(heads, _pad8(width), *w.shape[1:])
    out[:, :width] = w.reshape(heads, width, *w.shape[1:])
    return out.flatten(0, 1)


class FusedProjection:
    """Several projections of one input as one weight matrix; every part starts at a multiple of 8
    columns of the product (zero rows in between) and the input width is padded to a multiple of 8."""

    def __init__(self, parts, dtype, device):
        K = parts[0][1].shape[1]
        self.off, rows = {}, 0
        for name, w in parts:
            self.off[name] = rows
            rows += _pad8(w.shape[0])
        self.N, self.K = rows, _pad8(K)
        self.weight = torch.zeros(self.N, self.K, dtype=dtype, device=device)
        for name, w in parts:
            o = self.off[name]
            self.weight[o:o + w.shape[0], :K] = w.to(device=device, dtype=dtype)


class _Sublayer:
    """Norm weights around one sublayer."""

    def __init__(self, pre, post):
        self.pre, self.post = pre, post


class _Ctx:
    """One pass: token ids, the ragged batch (cu_q, kv_lens, slots, row_seq, pos), its block-table rows and sizes.
    ``decode``: one token of every sequence. ``split`` (passes with a long portion and latent layers):
    ``_LatentSplit``, else every token attends in the latent's space. ``conv``: what mixers read behind an input
    convolution."""

    def __init__(self, ids, batch, table, rows, n_seq, max_q, max_kv, split=None):
        self.ids, self.batch, self.table, self.rows, self.n_seq = ids, batch, table, rows, n_seq
        self.max_q, self.max_kv, self.split = max_q, max_kv, split
        self.decode = max_q == 1
        self.conv = None


class _LatentSplit:
    """Which tokens attend how: ``cu_k`` first expanded row of every sequence with a long portion (``keys`` in all,
    ``key_lens`` of each, at most ``max_k``), which holds its token ``first``; ``short`` the rows of the other sequences
    (None: there are none)."""

    def __init__(self, cu_k, first, key_lens, keys, max_k, short, short_seq, short_pos):
        self.cu_k, self.first, self.key_lens, self.keys, self.max_k = cu_k, first, key_lens, keys, max_k
        self.short, self.short_seq, self.short_pos = short, short_seq, short_pos


ACT_KINDS = {"silu": 0, "relu": 1, "clamped": 2}
DECODE_GEMM_ROWS = 128     # up to this many tokens a product goes through the few-token GEMM
EXPAND_TOKENS = 16         # portions of at least this many tokens expand the latents of their sequence
EXPAND_BYTES = 4 << 30     # unless the expanded keys and values would need more than this
SEGMENT_GEMM_ROWS = 48     # mean rows per expert from which the prompt-sized grouped GEMM runs
SIDE_STREAM_ROWS = 128     # up to this many tokens a parallel design's mixer and feed-forward run on two streams
LOW_RANK_FUSE_ROWS = 16    # decode batches up to this size evaluate the low-rank maps inside the recurrence kernel
STEP_FUSE_ROWS = 4         # the same for the step sizes of a selective scan, whose map every token reads again


class HybridEngine(InferenceEngine):
    paged_prefill_only = True
    # False: every step runs the plain any-shape kernels (token-by-token recurrence, scalar attention, one
    # kernel per step). Same results beyond rounding; for comparison and for 32-bit engines.
    tensor_kernels = True

    def __init__(self, cfg: HybridConfig, device="cuda", max_batch: int = 64, max_seq_len: int | None = None,
                 page_size: int = 16, tp=None, kv_pages: int | None = None, kv_dtype: str | None = None,
                 dtype: str = "bfloat16"):
        if tp is not None:
            raise ValueError("layer-list models run on one GPU")
        if kv_dtype not in (None, "bf16"):
            raise ValueError("layer-list models keep keys and values in the engine's activation type")
        if dtype not in DTYPES:
            raise ValueError(f"dtype must be one of {sorted(DTYPES)}, got {dtype!r}")
        self.cfg, self.device, self.tp = cfg, torch.device(device), None
        self.dtype = DTYPES[dtype]
        self.f32 = self.dtype == torch.float32
        self.max_batch = max_batch
        self.max_seq_len = min(max_seq_len or cfg.max_seq_len, cfg.context_limit)
        self.page_size = page_size
        self.world, self.rank = 1, 0
        pages_per_seq = (self.max_seq_len + page_size - 1) // page_size
        att = [s.attention for s in cfg.layers if s.attention is not None]
        recurrent = any(s.recurrent is not None for s in cfg.layers)
        self.states = RecurrentStatePool(max_batch, self.device) if recurrent or cfg.input_conv > 1 else None
        shapes = []                # per caching layer; a latent layer's rows are keys and values at once
        for s in cfg.layers:
            if s.attention is not None:
                if s.attention.kv_from is None:
                    shapes.append((s.attention.kv_heads, _pad8(s.attention.dim), _pad8(s.attention.vdim)))
            elif s.latent is not None and s.latent.kv_from is None:
                shapes.append((1, _pad8(s.latent.kv_rank) + _pad8(s.latent.rot_dim), 0))
        self.cache = PagedKVCache(len(shapes), 0, 0, kv_pages or max_batch * pages_per_seq, page_size, max_batch,
                                  pages_per_seq, self.device, dtype=self.dtype, layer_shapes=shapes, states=self.states)
        self.layers = []
        self.prefill_chunk = 8192
        self.prefill_chunk_threshold = 0
        self.last_prefix_hit = 0
        self._sms = torch.cuda.get_device_properties(self.device).multi_processor_count if self.device.type == "cuda" else 1
        self.H = native.require_hybrid() if self.device.type == "cuda" else None
        self._status = native.status_word(self.device)
        self._side = torch.cuda.Stream(self.device) if cfg.parallel and self.device.type == "cuda" else None
        groups = max([m.kv_heads * ((m.heads // m.kv_heads + 7) // 8) for m in att] or [1])
        self._counters = torch.zeros(max_batch * groups, device=self.device, dtype=torch.int32)
        experts = max([s.mlp.experts for s in cfg.layers if isinstance(s.mlp, MoeFF)] or [0])
        self._expert_counts = torch.zeros(experts + 1, device=self.device, dtype=torch.int32)
        self._max_ctx = self.max_seq_len

    # ------------------------------------------------------------------ weights
    @classmethod
    def from_model(cls, model, **kw) -> "HybridEngine":
        eng = cls(model.cfg, **kw)
        eng._pack(model)
        return eng

    @classmethod
    def random(cls, cfg, seed: int = 0, low_rank: int = 128, **kw) -> "HybridEngine":
        from ..models.hybrid import HybridModel

        eng = cls(cfg, **kw)
        eng._pack(HybridModel.random(cfg, seed, device=eng.device, dtype=torch.bfloat16, low_rank=low_rank))
        return eng

    def _matrix(self, w: torch.Tensor) -> torch.Tensor:
        """Weight matrix in the activation type, input width padded to a multiple of 8."""
        out = torch.zeros(w.shape[0], _pad8(w.shape[1]), dtype=self.dtype, device=self.device)
        out[:, : w.shape[1]] = w.to(device=self.device, dtype=self.dtype)
        return out

    def _vector(self, w: torch.Tensor) -> torch.Tensor:
        return w.to(device=self.device, dtype=torch.float32).contiguous()

    def _norm(self, w: torch.Tensor) -> torch.Tensor:
        return self._vector(w.expand(self.cfg.hidden_size) if w.dim() == 0 else w) + self.cfg.norm_offset

    def _pack(self, model) -> None:
        t = model.tensor
        cfg = self.cfg
        self.embed_table = t("embed").to(self.device, self.dtype).contiguous()
        self.pos_table = t("pos").to(self.device, self.dtype).contiguous() if cfg.position_table else None
        self.side_table = t("side.embed").to(self.device, self.dtype).contiguous() if cfg.token_side else None
        self.final_norm = self._norm(t("final.norm"))
        self.embed_norm = self._norm(t("embed.norm")) if cfg.embed_norm else None
        if not cfg.tied_head:
            self.head = self._matrix(t("head"))
        else:
            self.head = self.embed_table if cfg.hidden_size % 8 == 0 else self._matrix(self.embed_table)
        pages_of = {}                                 # layer -> its entry of the cache
        for i, spec in enumerate(cfg.layers):
            keeps = spec.attention or spec.latent
            share = keeps.kv_from if keeps is not None else None
            if share is not None:
                pages_of[i] = pages_of[share]
            elif keeps is not None:
                pages_of[i] = len(set(pages_of.values()))

        def norms(p: str, n: int) -> _Sublayer:
            if cfg.pre_norm:
                return _Sublayer(self._norm(t(p + f"norm{n}")), self._norm(t(p + f"norm{n}b")) if cfg.post_norm else None)
            return _Sublayer(None, self._norm(t(p + f"norm{n}")))

        for i, spec in enumerate(cfg.layers):
            p = f"l{i}."
            L = _HybridLayer()
            L.spec = spec
            L.norms = norms(p, 1)
            L.att_index = pages_of.get(i, 0)
            if isinstance(spec.mixer, ParallelMixer) and isinstance(spec.mixer.right, SelectiveMixer):
                L.run = self._parallel_selective
                self._pack_parallel_selective(L, t, p + "mix.")
            elif isinstance(spec.mixer, ParallelMixer):
                L.run = self._parallel
                self._pack_parallel(L, t, p + "mix.")
            elif isinstance(spec.mixer, AttentionMixer):
                L.run = self._attention_layer
                self._pack_attention(L, t, p + "mix.")
            elif isinstance(spec.mixer, LatentAttentionMixer):
                L.run = self._latent
                self._pack_latent(L, t, p + "mix.")
            else:
                L.run = self._gla
                self._pack_gla(L, t, p + "mix.")
            if cfg.input_conv:
                L.conv = self._input_conv(t(p + "canon1"))
            if cfg.parallel:
                self._pack_side_by_side(L, t, p + "mlp.")
            elif spec.mlp is not None:
                L.ff_norms = norms(p, 2)
                if isinstance(spec.mlp, MoeFF):
                    self._pack_experts(L, t, p + "mlp.")
                else:
                    L.act = (ACT_KINDS[spec.mlp.act], 0.0, 0.0)
                    self._pack_gated(L, t, p + "mlp.")
            if cfg.token_side:
                n = cfg.token_side
                L.side_gate, L.side_proj = self._matrix(t(p + "side.gate")), self._matrix(t(p + "side.proj"))
                L.side_embed = self.side_table[:, i * n:(i + 1) * n]
                L.side_norms = _Sublayer(None, self._vector(t(p + "side.norm")))
            self.layers.append(L)

    def _recurrent(self, m: RecurrentMixer, off: dict, tensors: dict):
        """Kernel-side object of one recurrence, with state of its own in the pool."""
        delta = m.kind == "delta"
        spec = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "taps": m.conv,
                "delta": int(delta), "unit_norm": int(delta), "decay_kind": int(delta), "gate_kind": int(delta),
                "q_scale": m.dim ** -0.5, "inv_tau": 1.0 / m.tau, "eps": self.cfg.norm_eps,
                **{k + "_off": v for k, v in off.items()}}
        tensors = dict(tensors)
        tensors["state"] = self.states.add(m.heads, m.vdim, m.dim)
        if m.conv > 1:
            tensors["conv_state"] = self.states.add(m.conv - 1, m.conv_channels)
        return self.H.Recurrent(spec, tensors)

    def _pack_gla(self, L, t, p: str) -> None:
        m = L.spec.mixer
        L.proj = FusedProjection([(n, t(p + n)) for n in ("q", "k", "v", "g", "a1")], self.dtype, self.device)
        L.a2, L.rank = self._matrix(t(p + "a2")), _pad8(t(p + "a1").shape[0])
        off = L.proj.off
        L.rec = self._recurrent(m, {"q": off["q"], "k": off["k"], "v": off["v"]},
                                {"z_bias": self._vector(t(p + "a2.b")), "gamma": self._vector(t(p + "norm")), "a2": L.a2})
        L.out = self._matrix(t(p + "o"))

    def _input_conv(self, w: torch.Tensor):
        channels, taps = w.shape
        return self.H.Conv(channels, True, self._vector(w.t()), state=self.states.add(taps - 1, channels) if taps > 1 else None)

    def _pack_side_by_side(self, L, t, p: str) -> None:
        """Feed-forward beside a mixer: its down matrix continues the rows of the mixer's output matrix."""
        mixer = L.run
        L.run, L.heads_of = self._side_by_side, {self._attention_layer: self._attention_heads, self._latent: self._latent_heads}[mixer]
        L.mixer_cols = L.out.shape[1]
        f = L.spec.mlp
        if f is None:
            return
        down = self._matrix(t(p + "down"))
        L.out = torch.cat([L.out, down], 1)
        L.down_bias = None
        if f.gated:
            L.gate_up = FusedProjection([("gate", t(p + "gate")), ("up", t(p + "up"))], self.dtype, self.device)
            L.act = (ACT_KINDS[f.act], 0.0, 0.0)
        else:
            L.up, L.up_bias = self._matrix(t(p + "up")), self._vector(t(p + "up.b"))
            L.poly, L.down_bias = self._vector(t(p + "act")), self._vector(t(p + "down.b"))

    # ---- attention: projection parts under a prefix, then the kernel-side object over their offsets
    def _attention_parts(self, m: AttentionMixer, t, p: str, prefix: str = "") -> list:
        parts = [("q", m.heads)]
        if m.kv_from is None:
            parts += [("k", m.kv_heads)] + ([("v", m.kv_heads)] if m.values == "own" else [])
        parts = [(prefix + n, _pad_heads(t(p + n), heads)) for n, heads in parts]
        if m.gate is not None:
            parts.append((prefix + "g", _pad_heads(t(p + "g"), m.heads) if m.gate == "channel" else t(p + "g")))
        return parts

    def _attention_object(self, m: AttentionMixer, t, p: str, off: dict, prefix: str = "", out_scale: float = 1.0):
        own = m.kv_from is None
        spec = {"heads": m.heads, "kv_heads": m.kv_heads, "dk": _pad8(m.dim), "dv": _pad8(m.vdim), "q_off": off[prefix + "q"],
                "scale": m.scale, "out_scale": out_scale, "window": m.window, "gate_channels": int(m.gate == "channel"),
                "norm_dim": m.dim if m.qk_norm else 0, "eps": self.cfg.norm_eps}
        if own:
            spec.update(k_off=off[prefix + "k"], v_off=off[prefix + ("v" if m.values == "own" else "k")])
        tensors = {}
        if m.bias:
            for n, heads in [("q", m.heads)] + ([("k", m.kv_heads), ("v", m.kv_heads)] if own else []):
                source = "k" if n == "v" and m.values == "keys" else n
                tensors[n + "_bias"] = self._vector(_pad_heads(t(p + source + ".b"), heads))
        if m.qk_norm == "weighted":
            for n in ("q", "k") if own else ("q",):
                tensors[n + "_gamma"] = self._vector(_pad_heads(t(p + n + ".norm"), 1))
        tensors.update(self._sink(m, t, p))
        if m.rotation is not None:
            spec.update(rot=m.rotation.dims, pairs=int(m.rotation.layout == "pairs"), rot_amp=m.rotation.amplitude)
            tensors["turns"] = torch.tensor(m.rotation.turns(), dtype=torch.float64, device=self.device)
        if m.q_temp is not None:
            spec.update(temp_coef=m.q_temp.coef, temp_every=m.q_temp.every)
        return self.H.Attention(spec, tensors)

    def _sink(self, m, t, p: str) -> dict:
        if m.sink is None:
            return {}
        return {"sink": self._vector(t(p + "sink")) if m.sink == "learned" else torch.zeros(m.heads, device=self.device)}

    @staticmethod
    def _attention_out(m: AttentionMixer, w: torch.Tensor) -> torch.Tensor:
        """Output matrix over padded value heads."""
        return _pad_heads(w.t(), m.heads).t()

    def _pack_attention(self, L, t, p: str) -> None:
        m = L.spec.attention
        L.proj = FusedProjection(self._attention_parts(m, t, p), self.dtype, self.device)
        L.att = self._attention_object(m, t, p, L.proj.off)
        L.out = self._matrix(self._attention_out(m, t(p + "o")))

    def _pack_parallel_selective(self, L, t, p: str) -> None:
        """Both mixers project from one GEMM and write their scaled outputs side by side for another."""
        a, r = L.spec.mixer.left, L.spec.mixer.right
        scale_l, scale_r = L.spec.mixer.scales
        left, right = p + "left.", p + "right."
        w_in, w_x = t(right + "in"), t(right + "x")
        L.proj = FusedProjection(self._attention_parts(a, t, left, "l") + [("rx", w_in[: r.inner]), ("rz", w_in[r.inner:])],
                                 self.dtype, self.device)
        L.att = self._attention_object(a, t, left, L.proj.off, "l", scale_l)
        n, k = r.state, r.dt_rank
        L.x_maps = FusedProjection([("dt", w_x[:k]), ("B", w_x[k:k + n]), ("C", w_x[k + n:])], self.dtype, self.device)
        L.w_dt = self._matrix(t(right + "dt"))
        padded = self.H.selective_padded_state(n)
        decay = torch.zeros(r.inner, padded, dtype=torch.float64)
        decay[:, :n] = -torch.exp(t(right + "A_log").double().cpu()) / math.log(2.0)
        tensors = {"a": self._vector(decay), "d": self._vector(t(right + "D")), "dt_b": self._vector(t(right + "dt.b")),
                   "w_dt": L.w_dt, "state": self.states.add(r.inner, padded)}
        L.conv = self.H.Conv(r.inner, False, self._vector(t(right + "conv").t()), self._vector(t(right + "conv.b")),
                             self.states.add(r.conv - 1, r.inner) if r.conv > 1 else None)
        L.sel = self.H.Selective({"inner": r.inner, "state": n, "rank": k, "out_scale": scale_r, "z_off": L.proj.off["rz"], "b_off": L.x_maps.off["B"],
                                  "c_off": L.x_maps.off["C"]}, tensors)
        L.out = self._matrix(torch.cat([self._attention_out(a, t(left + "o")), t(right + "o")], 1))

    def _pack_parallel(self, L, t, p: str) -> None:
        a, r = L.spec.mixer.left, L.spec.mixer.right
        left, right = p + "left.", p + "right."
        L.proj = FusedProjection(self._attention_parts(a, t, left, "l")
                                 + [("r" + n, t(right + n)) for n in ("q", "k", "v", "b", "a1", "g1")], self.dtype, self.device)
        L.att = self._attention_object(a, t, left, L.proj.off, "l")
        L.left_out, L.right_out = self._matrix(self._attention_out(a, t(left + "o"))), self._matrix(t(right + "o"))
        L.left_norm, L.right_norm = self._norm(t(left + "out")), self._norm(t(right + "out"))
        L.a2, L.rank = self._matrix(t(right + "a2")), _pad8(t(right + "a1").shape[0])
        L.g2, L.g_rank = self._matrix(t(right + "g2")), _pad8(t(right + "g1").shape[0])
        off = L.proj.off
        tensors = {"z_bias": self._vector(t(right + "dt_bias")), "a_log": self._vector(t(right + "A_log")),
                   "gamma": self._vector(t(right + "norm")), "a2": L.a2, "g2": L.g2}
        if r.conv > 0:
            tensors["conv_w"] = self._vector(torch.cat([t(right + n + ".conv") for n in ("q", "k", "v")]))
        L.rec = self._recurrent(r, {"q": off["rq"], "k": off["rk"], "v": off["rv"], "b": off["rb"]}, tensors)

    def _pack_latent(self, L, t, p: str) -> None:
        """Projection columns: unrotated queries per head | rotated queries per head (or, of low-rank queries, what a
        second matrix makes both from) | latent | rotated key part | gate, each part of a head padded to a multiple of 8."""
        m = L.spec.mixer
        H, dn, dr, dv, r = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        dn_p, dr_p, dv_p, r_p = _pad8(dn), _pad8(dr), _pad8(dv), _pad8(r)

        def heads(w, width, padded):                   # [heads * width, K] -> [heads * padded, K]
            out = w.new_zeros(H, padded, w.shape[1])
            out[:, :width] = w.view(H, width, -1)
            return out.view(H * padded, -1)

        order = torch.arange(dr)                       # rotated columns as neighbouring pairs
        if m.rotation.layout == "halves":
            order = torch.stack([order[: dr // 2], order[dr // 2:]], 1).flatten()
        q = t(p + ("uq" if m.q_rank else "q")).view(H, dn + dr, -1)
        queries = [("q", heads(q[:, :dn].reshape(H * dn, -1), dn, dn_p)),
                   ("qr", heads(q[:, dn:][:, order.to(q.device)].reshape(H * dr, -1), dr, dr_p))]
        parts = [("low", t(p + "dq"))] if m.q_rank else queries
        if m.kv_from is None:
            dkv = t(p + "dkv")
            parts = parts + [("c", dkv[:r]), ("kr", dkv[r:][order.to(dkv.device)])]
        if m.gate:
            parts = parts + [("g", heads(t(p + "g"), dv, dv_p))]
        L.proj = FusedProjection(parts, self.dtype, self.device)
        L.low = FusedProjection(queries, self.dtype, self.device) if m.q_rank else None
        uk, uv = t(p + "uk").view(H, dn, r), t(p + "uv").view(H, dv, r)
        L.uk_t = torch.zeros(H, r_p, dn_p, dtype=self.dtype, device=self.device)       # queries into the latent's space
        L.uk_t[:, :r, :dn] = uk.transpose(1, 2).to(self.device, self.dtype)
        L.uv = torch.zeros(H, dv_p, r_p, dtype=self.dtype, device=self.device)         # latents to a head's values
        L.uv[:, :dv, :r] = uv.to(self.device, self.dtype)
        off, own = L.proj.off, m.kv_from is None
        spec = {"heads": H, "rank": r, "rot": dr, "rank_p": r_p, "rot_p": dr_p, "qr_off": (L.low or L.proj).off["qr"],
                "scale": m.scale, "eps": self.cfg.norm_eps, "window": m.window, "rot_amp": m.rotation.amplitude}
        if own:
            spec.update(c_off=off["c"], kr_off=off["kr"])
        if m.q_rank:
            spec.update(low_off=off["low"], low_rank=m.q_rank)
        turns = torch.tensor(m.rotation.turns(), dtype=torch.float64, device=self.device)
        L.lat = self.H.Latent(spec, self._vector(t(p + "dkv.norm")) if own else None, turns, self._sink(m, t, p).get("sink"),
                              self._vector(t(p + "dq.norm")) if m.q_rank else None)
        L.expand = None
        if self.tensor_kernels and not self.f32 and L.lat.prefill_ok(dn_p, dv_p):      # keys and values of all heads
            L.expand = torch.zeros(H * (dn_p + dv_p), r_p, dtype=self.dtype, device=self.device)
            L.expand[: H * dn_p].view(H, dn_p, r_p)[:, :dn, :r] = uk.to(self.device, self.dtype)
            L.expand[H * dn_p:].view(H, dv_p, r_p).copy_(L.uv)
        out = t(p + "o")
        w = out.new_zeros(out.shape[0], H, dv_p)
        w[:, :, :dv] = out.view(-1, H, dv)
        L.out = self._matrix(w.view(-1, H * dv_p))

    def _pack_gated(self, L, t, p: str) -> None:
        L.gate_up = FusedProjection([("gate", t(p + "gate")), ("up", t(p + "up"))], self.dtype, self.device)
        L.down = self._matrix(t(p + "down"))

    def _pack_experts(self, L, t, p: str) -> None:
        """Gate and up rows of an expert in one matrix [2 * ff, d], all experts stacked; ff padded to a multiple of 8."""
        m, d = L.spec.mlp, self.cfg.hidden_size
        f = _pad8(m.ff)
        L.act = (ACT_KINDS[m.act], m.limit, m.alpha)
        L.router, L.correction = self._matrix(t(p + "router")), self._vector(t(p + "correction")) if m.correction else None
        L.rule = (int(m.score == "sigmoid"), m.group_best, int(m.normalise), m.scale)
        if m.shared:
            self._pack_gated(L, t, p + "shared.")
        L.w_in = torch.zeros(m.experts, 2 * f, _pad8(d), dtype=self.dtype, device=self.device)
        L.w_out = torch.zeros(m.experts, _pad8(d), f, dtype=self.dtype, device=self.device)
        for e in range(m.experts):
            L.w_in[e, : m.ff, :d] = t(p + f"e{e}.gate").to(self.device, self.dtype)
            L.w_in[e, f:f + m.ff, :d] = t(p + f"e{e}.up").to(self.device, self.dtype)
            L.w_out[e, :d, : m.ff] = t(p + f"e{e}.down").to(self.device, self.dtype)

    def weight_bytes(self) -> int:
        tables = (self.embed_table, self.pos_table, self.side_table, self.head if self.head is not self.embed_table else None)
        n = sum(x.numel() * x.element_size() for x in tables if x is not None)
        for L in self.layers:
            mats = [L.proj.weight, L.a2, L.g2, L.out, L.left_out, L.right_out, L.down, L.uk_t, L.uv, L.router, L.w_in, L.w_out,
                    L.side_gate, L.side_proj, L.w_dt, L.up] + [f.weight for f in (L.gate_up, L.x_maps, L.low) if f is not None]
            n += sum(x.numel() * x.element_size() for x in mats if x is not None)
        return n

    # ------------------------------------------------------------------ pieces of a pass
    def _new(self, rows: int, cols: int, dtype=None) -> torch.Tensor:
        return torch.empty(rows, cols, device=self.device, dtype=dtype or self.dtype)

    def _gemm(self, x, w, out=None, dtype=None, alpha: float = 1.0, cap: float = 0.0):
        """alpha * x w^T; with ``cap`` (fp32 results) the soft-capped product."""
        if out is None:
            out = self._new(x.shape[0], w.shape[0], dtype)
        if self._fast and x.shape[0] <= DECODE_GEMM_ROWS:
            self.H.gemm_decode(x, w, out, 0, 0, alpha, self._status, cap=cap)
        else:
            self.H.gemm_nt(x, w, out, alpha, self._status)
            if cap > 0.0:
                self.H.soft_cap(out, cap)
        return out

    @property
    def _fast(self) -> bool:
        return self.tensor_kernels and not self.f32

    def _recurrence(self, L, proj, a_off: int, gate, g_off: int, ctx):
        """Recurrence of a layer over the batch, head norm and output gate -> [rows, pad8(heads * vdim)].
        ``a_off`` / ``g_off``: columns of ``proj`` with the inner products of the low-rank maps of the decay
        and (where ``gate`` is None) of the output gate."""
        m, rec = L.spec.recurrent, L.rec
        out = self._new(ctx.rows, _pad8(m.heads * m.vdim))
        fuse = ctx.decode and self.tensor_kernels and ctx.rows <= LOW_RANK_FUSE_ROWS
        z = None
        if not fuse:
            z = self._gemm(proj[:, a_off:a_off + L.rank], L.a2, dtype=torch.float32)
            if gate is None:
                gate = self._gemm(proj[:, g_off:g_off + L.g_rank], L.g2)
        if ctx.decode and self.tensor_kernels:
            rec.decode(proj, z, gate, a_off, g_off, ctx.batch, out)
            return out
        o = torch.empty(ctx.rows, m.heads, m.vdim, device=self.device, dtype=torch.float32)
        if self._fast and rec.chunked_ok():
            scratch = torch.empty(rec.chunked_scratch(ctx.rows, ctx.n_seq), device=self.device, dtype=torch.uint8)
            rec.scan_chunked(proj, z, ctx.batch, scratch, o, self._status)
        else:
            scratch = torch.empty(ctx.rows * (2 * m.kv_heads * m.dim + m.heads * (m.vdim + m.dim + 1)),
                                  device=self.device, dtype=torch.float32)
            rec.scan_seq(proj, z, ctx.batch, scratch, o)
        rec.norm_gate(o, gate, out)
        return out

    def _gla(self, L, h, ctx):
        off = L.proj.off
        proj = self._gemm(h, L.proj.weight)
        y = self._recurrence(L, proj, off["a1"], proj[:, off["g"]:], 0, ctx)
        return self._gemm(y, L.out), None

    def _attention(self, L, proj, ctx, prefix: str = "", out=None):
        """Attention up to its output projection -> [rows, heads * padded value width]."""
        m, att = L.spec.attention, L.att
        kc, vc = self.cache.k[L.att_index], self.cache.v[L.att_index]
        dk, dv = kc.shape[3], vc.shape[3]
        q = torch.empty(ctx.rows, m.heads, dk, device=self.device, dtype=self.dtype)
        att.prep(proj, ctx.batch, ctx.table, q, kc, vc)
        o = self._new(ctx.rows, m.heads * dv) if out is None else out
        gate = None
        if m.gate is not None:
            g = L.proj.off[prefix + "g"]
            gate = proj[:, g:g + m.heads * (dv if m.gate == "channel" else 1)]
        if not (self._fast and att.tensor_ok(self.page_size)):
            att.any(q, kc, vc, ctx.batch, ctx.table, gate, o)
        elif ctx.decode:
            keys = min(ctx.max_kv, m.window + self.page_size) if m.window else ctx.max_kv
            pairs = ctx.n_seq * m.kv_heads * ((m.heads // m.kv_heads + 7) // 8)
            splits = max(1, min(32, (6 * self._sms + pairs - 1) // pairs, (keys + 255) // 256))
            scratch = torch.empty(att.decode_scratch(ctx.rows, splits), device=self.device, dtype=torch.float32)
            att.decode(q, kc, vc, ctx.batch, ctx.table, gate, o, scratch, self._counters, splits, self._status)
        else:
            att.prefill(q, kc, vc, ctx.batch, ctx.table, gate, o, ctx.max_q, self._status)
        return o

    def _attention_heads(self, L, h, ctx, out=None):
        return self._attention(L, self._gemm(h, L.proj.weight), ctx, out=out)

    def _attention_layer(self, L, h, ctx):
        return self._gemm(self._attention_heads(L, h, ctx), L.out), None

    def _selective(self, L, proj, ctx, out):
        """Selective scan of a layer over the batch with its output gate -> out [rows, padded channels]."""
        m, sel = L.spec.recurrent, L.sel
        one = ctx.decode and self.tensor_kernels
        x = self._new(ctx.rows, _pad8(m.inner))
        L.conv.run(proj, L.proj.off["rx"], ctx.batch, one, x)
        low = self._gemm(x, L.x_maps.weight)
        dt = None
        if not (one and ctx.rows <= STEP_FUSE_ROWS):
            dt = self._gemm(low[:, : L.w_dt.shape[1]], L.w_dt, dtype=torch.float32)
        if out.shape[1] != m.inner:
            out[:, m.inner:].zero_()
        if one:
            sel.step(proj, x, low, dt, ctx.batch, out)
        else:
            scratch = torch.empty(sel.scratch_floats(ctx.n_seq, ctx.rows, ctx.max_q), device=self.device, dtype=torch.float32)
            sel.scan(proj, x, low, dt, ctx.batch, ctx.max_q, scratch, out, self._status)

    def _parallel_selective(self, L, h, ctx):
        proj = self._gemm(h, L.proj.weight)
        y = self._new(ctx.rows, L.out.shape[1])
        n = L.spec.attention.heads * self.cache.v[L.att_index].shape[3]
        self._attention(L, proj, ctx, "l", y[:, :n])
        self._selective(L, proj, ctx, y[:, n:])
        return self._gemm(y, L.out), None

    def _parallel(self, L, h, ctx):
        off = L.proj.off
        proj = self._gemm(h, L.proj.weight)
        y_right = self._gemm(self._recurrence(L, proj, off["ra1"], None, off["rg1"], ctx), L.right_out)
        y_left = self._gemm(self._attention(L, proj, ctx, "l"), L.left_out)
        return y_left, y_right

    # ---- latent attention
    def _latent_tokens(self, L, queries, gate, row_seq, pos, ctx, out=None):
        """Tokens that attend in the latent's space -> [rows, heads, padded value width]."""
        m, H = L.spec.mixer, L.spec.mixer.heads
        n, cache = queries.shape[0], self.cache.k[L.att_index]
        r_p, dn_p = L.uk_t.shape[1:]
        q = queries[:, : H * dn_p].unflatten(1, (H, dn_p))
        q_lat = torch.empty(n, H, r_p, device=self.device, dtype=self.dtype)
        o_lat = torch.empty_like(q_lat)
        self.H.gemm_heads(q, L.uk_t, q_lat, self._status)
        if self._fast and L.lat.decode_ok(self.page_size):
            splits = self._latent_splits(n, H, min(ctx.max_kv, m.window + 64) if m.window else ctx.max_kv)
            scratch = torch.empty(n * H * splits * (r_p + 4) if splits > 1 else 0, device=self.device, dtype=torch.float32)
            L.lat.attn_decode(q_lat, queries, row_seq, pos, ctx.table, cache, o_lat, scratch, splits, self._status)
        else:
            L.lat.attn_any(q_lat, queries, row_seq, pos, ctx.table, cache, o_lat)
        if out is None:
            out = torch.empty(n, H, L.uv.shape[1], device=self.device, dtype=self.dtype)
        self.H.gemm_heads(o_lat, L.uv, out, self._status, gate)
        return out

    def _latent_splits(self, rows: int, heads: int, max_kv: int) -> int:
        """At most one CTA per SM (a CTA fills one), and two 64-token tiles of work for each."""
        pairs = rows * ((heads + 15) // 16)
        return max(1, min(64, self._sms // pairs, (max_kv + 127) // 128))

    def _latent_heads(self, L, h, ctx, out=None):
        """Latent attention up to its output projection -> [rows, heads * padded value width]."""
        m, H = L.spec.mixer, L.spec.mixer.heads
        proj = self._gemm(h, L.proj.weight)
        cache = self.cache.k[L.att_index]
        queries = proj
        if L.low is not None:                          # the vector that both query parts are a map of comes first
            L.lat.prep(proj, ctx.batch, ctx.table, cache, queries=False)
            queries = self._gemm(proj[:, : L.low.K], L.low.weight)
        L.lat.prep(queries, ctx.batch, ctx.table, cache, latents=L.low is None)
        dn_p, dv_p = L.uk_t.shape[2], L.uv.shape[1]
        gate = proj[:, L.proj.off["g"]:][:, : H * dv_p] if m.gate else None
        if out is None:
            out = self._new(ctx.rows, H * dv_p)
        o = out.unflatten(1, (H, dv_p))
        sp = ctx.split
        if sp is None or L.expand is None or not self._fast or sp.keys * L.expand.shape[0] * 2 > EXPAND_BYTES:
            self._latent_tokens(L, queries, gate, ctx.batch[3], ctx.batch[4], ctx, o)
            return out
        latents = self._new(sp.keys, cache.shape[3])
        L.lat.gather(ctx.table, cache, sp.cu_k, sp.first, sp.max_k, latents)
        kv = self._gemm(latents[:, : L.expand.shape[1]], L.expand)
        L.lat.attn_prefill(queries[:, : H * dn_p].unflatten(1, (H, dn_p)), queries, kv[:, : H * dn_p].unflatten(1, (H, dn_p)),
                           kv[:, H * dn_p:].unflatten(1, (H, dv_p)), latents, ctx.batch, sp.cu_k, sp.key_lens, ctx.max_q,
                           EXPAND_TOKENS, gate, o, self._status)
        if sp.short is not None:
            o.index_copy_(0, sp.short, self._latent_tokens(L, queries.index_select(0, sp.short),
                                                           gate.index_select(0, sp.short) if gate is not None else None,
                                                           sp.short_seq, sp.short_pos, ctx))
        return out

    def _latent(self, L, h, ctx):
        return self._gemm(self._latent_heads(L, h, ctx), L.out), None

    # ---- feed-forwards
    def _expert_tile(self, rows: int, m) -> int:
        """Rows of a tile of the grouped GEMMs, from the mean rows per expert."""
        mean = rows * m.top // m.experts
        if self.f32:
            return 64
        return 128 if mean >= SEGMENT_GEMM_ROWS else max(16, min(64, 1 << (2 * mean).bit_length()))

    def _experts(self, L, h, ctx):
        """Outputs of the chosen experts [rows * top, d], of the shared expert, where each (token, choice) lies and its
        weight."""
        m, T, C = L.spec.mlp, ctx.rows, self.H
        z = self._gemm(h, L.router, dtype=torch.float32)
        pairs, tile = T * m.top, self._expert_tile(T, m)
        i32 = dict(device=self.device, dtype=torch.int32)
        idx, slot, row = (torch.empty(T, m.top, **i32) for _ in range(3))
        weight = torch.empty(T, m.top, device=self.device, dtype=torch.float32)
        offset, count = torch.empty(m.experts, **i32), torch.empty(1, **i32)
        tiles = torch.empty(min(pairs, m.experts + pairs // tile), 3, **i32)
        route = (m.experts, m.top, m.groups, m.keep)
        plan = (idx, weight, slot, self._expert_counts[: m.experts + 1], offset, tiles, count)
        C.expert_select(z, L.correction, route, tile, *plan, L.rule)
        d_p, f = L.w_in.shape[2], L.w_out.shape[2]
        x = self._new(pairs, d_p)
        C.expert_gather(h, route, *plan, x, row)
        a, y = self._new(pairs, f), self._new(pairs, d_p)
        if self.f32:
            gu = self._new(pairs, 2 * f)
            C.gemm_tiles(x, L.w_in, gu, tiles, count, tile, 0, 0, L.act, self._status)
            C.gate_pair(gu, f, f, L.act, a)
        else:
            C.gemm_tiles(x, L.w_in, a, tiles, count, tile, f, f, L.act, self._status)
        C.gemm_tiles(a, L.w_out, y, tiles, count, tile, 0, 0, L.act, self._status)
        shared = None
        if m.shared:
            shared = self._new(T, d_p)
            self._gated(L, m.shared, h, ctx, shared[:, : self.cfg.hidden_size])
        return y, shared, row, weight

    def _gated(self, L, f: int, h, ctx, out=None):
        """Gated feed-forward of width ``f`` for every token."""
        a = self._new(ctx.rows, L.down.shape[1])
        if self._fast and f % 8 == 0 and ctx.rows <= DECODE_GEMM_ROWS:
            self.H.gemm_decode(h, L.gate_up.weight, a, f, L.gate_up.off["up"], 1.0, self._status, L.act)
        elif self._fast and L.act[0] == 0 and f % 128 == 0 and ctx.rows >= 256:
            self.H.gemm_swiglu(h, L.gate_up.weight, a, self._status)
        else:
            gu = self._gemm(h, L.gate_up.weight)
            self.H.gate_pair(gu, f, L.gate_up.off["up"], L.act, a)
        return self._gemm(a, L.down, out)

    def _ff_columns(self, L, h, out):
        """Feed-forward up to its down matrix."""
        if L.up is not None:
            self.H.poly_norm(self._gemm(h, L.up), L.up_bias, L.poly, L.spec.mlp.ff, out, self.cfg.norm_eps)
        elif L.gate_up is not None:
            gu, a = self._gemm(h, L.gate_up.weight), self._new(*out.shape)
            self.H.gate_pair(gu, L.spec.mlp.ff, L.gate_up.off["up"], L.act, a)
            out.copy_(a)

    def _side_by_side(self, L, h, ctx):
        """Mixer and feed-forward of a parallel design -> their sum. Few tokens leave most of the GPU idle: the two run
        on streams of their own."""
        y = self._new(ctx.rows, L.out.shape[1])
        n = L.mixer_cols
        mixer_in = ctx.conv if L.conv is not None else h
        if ctx.rows <= SIDE_STREAM_ROWS and L.spec.mlp is not None:
            main = torch.cuda.current_stream(self.device)
            self._side.wait_stream(main)
            with torch.cuda.stream(self._side):
                self._ff_columns(L, h, y[:, n:])
            L.heads_of(L, mixer_in, ctx, y[:, :n])
            main.wait_stream(self._side)
        else:
            L.heads_of(L, mixer_in, ctx, y[:, :n])
            self._ff_columns(L, h, y[:, n:])
        return self._gemm(y, L.out)

    def _feed_forward(self, L, h, ctx):
        return self._gated(L, L.spec.mlp.ff, h, ctx)

    def _token_side(self, L, h, ctx):
        """proj(gelu(gate x) * side embedding of the token)"""
        g = self._new(ctx.rows, L.side_proj.shape[1])
        n = L.side_gate.shape[0]
        if g.shape[1] != n:
            g[:, n:].zero_()
        if self._fast:
            self.H.gemm_decode(h, L.side_gate, g, 0, 0, 1.0, self._status, (0, 0.0, 0.0), L.side_embed, ctx.ids)
        else:
            self.H.gemm_nt(h, L.side_gate, g[:, :n], 1.0, self._status)
            self.H.gelu_mul(g[:, :n], L.side_embed, ctx.ids)
        return self._gemm(g, L.side_proj)

    # ------------------------------------------------------------------ the pass
    def _paged_prefill_ok(self) -> bool:
        return True

    def _prepare_decode_scratch(self, batch: int, max_ctx: int):
        self._max_ctx = max_ctx

    def _forward(self, ids, pos, seq_ids, ctx_lens, prefill_shape=None, paged=None):
        """``paged`` as in the base class; without it every row is one token of the sequence ``seq_ids[row]``
        with ``ctx_lens[row]`` tokens including it (a decode step)."""
        if paged is not None:
            cu_q, kv_lens, table, max_q, slots, row_seq, max_kv, split = paged
        else:
            n = ids.numel()
            cu_q = torch.arange(n + 1, device=self.device, dtype=torch.int32)
            row_seq, slots, kv_lens, max_q, max_kv, split = cu_q[:n], seq_ids, ctx_lens, 1, self._max_ctx, None
            table = self.cache.block_table.index_select(0, slots)
        ctx = _Ctx(ids, [cu_q, kv_lens, slots, row_seq, pos], table, ids.numel(), kv_lens.numel(), max_q, max_kv, split)
        return self._run_layers(ids, pos, ctx)

    def _batch_plan(self, lens, bases):
        windows = [s.latent.window for s in self.cfg.layers if s.latent is not None]
        if not windows or max(lens) < EXPAND_TOKENS:
            return [], None
        reach = max(windows) if min(windows) > 0 else 0        # keys in front of a query that some layer sees, 0: all
        cu_k, first, key_lens, short, short_seq, short_pos, at = [0], [], [], [], [], [], 0
        for i, (n, base) in enumerate(zip(lens, bases)):
            first.append(max(0, base - reach + 1) if reach and n >= EXPAND_TOKENS else 0)
            key_lens.append(base + n - first[-1])
            if n >= EXPAND_TOKENS:
                cu_k.append(cu_k[-1] + key_lens[-1])
            else:
                cu_k.append(cu_k[-1])
                short += range(at, at + n)
                short_seq += [i] * n
                short_pos += range(base, base + n)
            at += n

        max_k = max(b - a for a, b in zip(cu_k, cu_k[1:]))

        def build(cu, skipped, keys, rows, seq, pos):
            return _LatentSplit(cu, skipped, keys, cu_k[-1], max_k, rows.long() if short else None, seq, pos)

        return [cu_k, first, key_lens, short, short_seq, short_pos], build

    def _run_layers(self, ids, pos, ctx, trace=None):
        cfg, H = self.cfg, self.H
        d, eps = cfg.hidden_size, cfg.norm_eps
        x = self._new(ctx.rows, d, torch.float32)
        h = self._new(ctx.rows, _pad8(d))
        if cfg.input_conv:
            ctx.conv = self._new(ctx.rows, _pad8(d))
        subs = []                                    # (layer, sublayer function, its norms)
        for L in self.layers:
            subs.append((L, L.run, L.norms))
            if L.spec.mlp is not None and not cfg.parallel:
                subs.append((L, self._experts if L.router is not None else self._feed_forward, L.ff_norms))
            if L.side_gate is not None:
                subs.append((L, self._token_side, L.side_norms))

        def conv_tail(j):                            # single tokens: the kernel that writes h runs sublayer j's convolution
            return (subs[j][0].conv, ctx.batch, ctx.conv) if cfg.input_conv and ctx.decode and j < len(subs) else None

        H.embed_pos_norm(ids, pos, self.embed_table, self.pos_table, cfg.embed_scale,
                         subs[0][2].pre if subs else self.final_norm, x, h, eps, self.embed_norm, conv_tail(0))
        for j, (L, fn, norms) in enumerate(subs):
            nxt = subs[j + 1][2].pre if j + 1 < len(subs) else self.final_norm
            if cfg.input_conv and not ctx.decode:
                L.conv.run(h, 0, ctx.batch, False, ctx.conv)
            y = fn(L, h, ctx)
            if cfg.parallel:
                H.residual_norm(y, L.down_bias, cfg.residual_mult, x, nxt, h, eps, conv_tail(j + 1))
            elif fn == self._experts:
                H.expert_norm(*y, norms.post, x, nxt, h, eps, cfg.residual_mult)
            else:
                y1, y2 = y if isinstance(y, tuple) else (y, None)
                H.sandwich_norm(y1, y2, L.left_norm, L.right_norm, norms.post, x, nxt, h, eps, cfg.residual_mult)
            if trace is not None and (j + 1 == len(subs) or subs[j + 1][0] is not L):
                trace.append(x.clone())
        return h

    def _decode_rows(self, ids, pos, sid):
        return self._forward(ids, pos, sid, pos + 1)

    def _logits(self, h):
        if h.shape[1] != self.head.shape[1] or h.dtype != self.dtype:
            full = torch.zeros(h.shape[0], self.head.shape[1], device=self.device, dtype=self.dtype)
            full[:, : h.shape[1]] = h
            h = full
        return self._gemm(h, self.head, dtype=torch.float32, alpha=self.cfg.logit_scale, cap=self.cfg.logit_softcap)


class _HybridLayer:
    spec = norms = ff_norms = proj = a2 = g2 = out = left_out = right_out = left_norm = right_norm = rec = None
    att = sel = x_maps = w_dt = None
    conv = low = up = up_bias = poly = down_bias = heads_of = None
    mixer_cols = 0
    gate_up = down = act = router = correction = rule = w_in = w_out = None
    lat = uk_t = uv = expand = run = None
    side_gate = side_proj = side_embed = side_norms = None
    rank = g_rank = att_index = 0

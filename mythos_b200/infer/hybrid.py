"""Inference engine of layer-list models (:mod:`mythos_b200.models.hybrid_config`).

``HybridEngine`` is an :class:`InferenceEngine`: generation, the step-wise API, sampling, the page
allocator and the CUDA-graph decode loop are the base class's. It brings its own pass over the layers
and, beside the attention layers' pages, a slot of recurrent state per sequence.

A pass takes a ragged batch (new tokens of several sequences, packed; prompts, portions of prompts and
single decoded tokens in any mix). The residual stream is fp32; a sublayer reads its normalised copy in
the engine's activation type. All projections of a mixer that read the same input are one GEMM. Per
gated-linear-attention layer: projections -> decay GEMM -> recurrence -> head norm * gate -> output
GEMM -> (post-norm + residual + next pre-norm). A parallel layer runs the delta-rule recurrence and
paged attention side by side and averages their normalised outputs inside that last kernel.

``dtype``: "bfloat16" (matrix products and activations in bf16 with 32-bit accumulation; residual,
norms, decays, states and scores in 32-bit) or "float32" (everything in 32-bit).
"""
from __future__ import annotations

import torch

from ..models.hybrid_config import HybridConfig, ParallelMixer, RecurrentMixer
from ..ops import native
from .engine import InferenceEngine
from .kv_paged import PagedKVCache, RecurrentStatePool

DTYPES = {"bfloat16": torch.bfloat16, "bf16": torch.bfloat16, "float32": torch.float32, "fp32": torch.float32}


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


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
    """One pass: the ragged batch (cu_q, kv_lens, slots, row_seq, pos), its block-table rows and sizes.
    ``decode``: one token of every sequence."""

    def __init__(self, batch, table, rows, n_seq, max_q, max_kv):
        self.batch, self.table, self.rows, self.n_seq, self.max_q, self.max_kv = batch, table, rows, n_seq, max_q, max_kv
        self.decode = max_q == 1


DECODE_GEMM_ROWS = 128     # up to this many tokens a product goes through the few-token GEMM
LOW_RANK_FUSE_ROWS = 16    # decode batches up to this size evaluate the low-rank maps inside the recurrence kernel


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
        self.max_seq_len = min(max_seq_len or cfg.max_seq_len, cfg.max_seq_len)
        self.page_size = page_size
        self.world, self.rank = 1, 0
        pages_per_seq = (self.max_seq_len + page_size - 1) // page_size
        att = [s.attention for s in cfg.layers if s.attention is not None]
        self.states = RecurrentStatePool(max_batch, self.device)
        self.cache = PagedKVCache(len(att), 0, 0, kv_pages or max_batch * pages_per_seq, page_size, max_batch,
                                  pages_per_seq, self.device, dtype=self.dtype,
                                  layer_shapes=[(m.kv_heads, m.dim, m.vdim) for m in att], states=self.states)
        self.layers = []
        self.prefill_chunk = 8192
        self.prefill_chunk_threshold = 0
        self.last_prefix_hit = 0
        self._sms = torch.cuda.get_device_properties(self.device).multi_processor_count if self.device.type == "cuda" else 1
        self.H = native.require_hybrid() if self.device.type == "cuda" else None
        self._status = native.status_word(self.device)
        groups = max([m.kv_heads * ((m.heads // m.kv_heads + 7) // 8) for m in att] or [1])
        self._counters = torch.zeros(max_batch * groups, device=self.device, dtype=torch.int32)
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

    def _pack(self, model) -> None:
        t = model.tensor
        self.embed_table = t("embed").to(self.device, self.dtype).contiguous()
        self.pos_table = t("pos").to(self.device, self.dtype).contiguous()
        self.final_norm = self._vector(t("final.norm"))
        self.head = self._matrix(t("head"))
        n_att = 0
        for i, spec in enumerate(self.cfg.layers):
            p = f"l{i}."
            L = _HybridLayer()
            L.spec = spec
            L.norms = _Sublayer(self._vector(t(p + "norm1")), self._vector(t(p + "norm1b")))
            if isinstance(spec.mixer, ParallelMixer):
                self._pack_parallel(L, t, p + "mix.", n_att)
                n_att += 1
            else:
                self._pack_gla(L, t, p + "mix.")
            if spec.ff:
                L.ff_norms = _Sublayer(self._vector(t(p + "norm2")), self._vector(t(p + "norm2b")))
                L.gate_up = FusedProjection([("gate", t(p + "mlp.gate")), ("up", t(p + "mlp.up"))], self.dtype, self.device)
                L.down = self._matrix(t(p + "mlp.down"))
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

    def _pack_parallel(self, L, t, p: str, att_index: int) -> None:
        a, r = L.spec.mixer.left, L.spec.mixer.right
        left, right = p + "left.", p + "right."
        L.proj = FusedProjection(
            [("lq", t(left + "q")), ("lk", t(left + "k")), ("lv", t(left + "v")), ("lg", t(left + "g"))]
            + [("r" + n, t(right + n)) for n in ("q", "k", "v", "b", "a1", "g1")], self.dtype, self.device)
        L.att_index = att_index
        L.q_gamma, L.k_gamma = self._vector(t(left + "q.norm")), self._vector(t(left + "k.norm"))
        L.left_out, L.right_out = self._matrix(t(left + "o")), self._matrix(t(right + "o"))
        L.left_norm, L.right_norm = self._vector(t(left + "out")), self._vector(t(right + "out"))
        L.a2, L.rank = self._matrix(t(right + "a2")), _pad8(t(right + "a1").shape[0])
        L.g2, L.g_rank = self._matrix(t(right + "g2")), _pad8(t(right + "g1").shape[0])
        off = L.proj.off
        tensors = {"z_bias": self._vector(t(right + "dt_bias")), "a_log": self._vector(t(right + "A_log")),
                   "gamma": self._vector(t(right + "norm")), "a2": L.a2, "g2": L.g2}
        if r.conv > 0:
            tensors["conv_w"] = self._vector(torch.cat([t(right + n + ".conv") for n in ("q", "k", "v")]))
        L.rec = self._recurrent(r, {"q": off["rq"], "k": off["rk"], "v": off["rv"], "b": off["rb"]}, tensors)

    def weight_bytes(self) -> int:
        n = sum(x.numel() * x.element_size() for x in (self.embed_table, self.pos_table, self.head))
        for L in self.layers:
            mats = [L.proj.weight, L.a2, L.g2, L.out, L.left_out, L.right_out, L.down,
                    L.gate_up.weight if L.gate_up is not None else None]
            n += sum(x.numel() * x.element_size() for x in mats if x is not None)
        return n

    # ------------------------------------------------------------------ pieces of a pass
    def _new(self, rows: int, cols: int, dtype=None) -> torch.Tensor:
        return torch.empty(rows, cols, device=self.device, dtype=dtype or self.dtype)

    def _gemm(self, x, w, out=None, dtype=None, alpha: float = 1.0):
        if out is None:
            out = self._new(x.shape[0], w.shape[0], dtype)
        if self._fast and x.shape[0] <= DECODE_GEMM_ROWS:
            self.H.gemm_decode(x, w, out, 0, 0, alpha, self._status)
        else:
            self.H.gemm_nt(x, w, out, alpha, self._status)
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

    def _attention(self, L, proj, ctx):
        """Left mixer of a parallel layer up to its output projection."""
        m, off, li = L.spec.attention, L.proj.off, L.att_index
        kc, vc = self.cache.k[li], self.cache.v[li]
        q = torch.empty(ctx.rows, m.heads, m.dim, device=self.device, dtype=self.dtype)
        self.H.qk_norm_append(proj, off["lq"], off["lk"], off["lv"], L.q_gamma, L.k_gamma, ctx.batch, ctx.table, q, kc, vc,
                              self.cfg.norm_eps)
        width = m.heads * m.vdim
        o = self._new(ctx.rows, _pad8(width))
        if o.shape[1] != width:
            o[:, width:].zero_()
        gate = proj[:, off["lg"]:off["lg"] + m.heads]
        if not (self._fast and self.page_size == 16 and m.dim in (64, 128) and m.vdim in (64, 128)):
            self.H.paged_attn_any(q, kc, vc, ctx.batch, ctx.table, gate, o, m.scale)
        elif ctx.decode:
            pairs = ctx.n_seq * m.kv_heads * ((m.heads // m.kv_heads + 7) // 8)
            splits = max(1, min(32, (6 * self._sms + pairs - 1) // pairs, (ctx.max_kv + 255) // 256))
            scratch = torch.empty(ctx.rows * m.heads * splits * (m.vdim + 2), device=self.device, dtype=torch.float32)
            self.H.paged_attn_decode(q, kc, vc, ctx.batch, ctx.table, gate, o, scratch, self._counters, splits, m.scale,
                                     self._status)
        else:
            self.H.paged_attn_prefill(q, kc, vc, ctx.batch, ctx.table, gate, o, ctx.max_q, m.scale, self._status)
        return o

    def _parallel(self, L, h, ctx):
        off = L.proj.off
        proj = self._gemm(h, L.proj.weight)
        y_right = self._gemm(self._recurrence(L, proj, off["ra1"], None, off["rg1"], ctx), L.right_out)
        y_left = self._gemm(self._attention(L, proj, ctx), L.left_out)
        return y_left, y_right

    def _feed_forward(self, L, h, ctx):
        f = L.spec.ff
        a = self._new(ctx.rows, L.down.shape[1])
        if self._fast and f % 8 == 0 and ctx.rows <= DECODE_GEMM_ROWS:
            self.H.gemm_decode(h, L.gate_up.weight, a, f, L.gate_up.off["up"], 1.0, self._status)
            return self._gemm(a, L.down)
        if self._fast and f % 128 == 0 and ctx.rows >= 256:
            self.H.gemm_swiglu(h, L.gate_up.weight, a, self._status)
            return self._gemm(a, L.down)
        gu = self._gemm(h, L.gate_up.weight)
        self.H.silu_gate(gu, f, L.gate_up.off["up"], a)
        return self._gemm(a, L.down)

    # ------------------------------------------------------------------ the pass
    def _paged_prefill_ok(self) -> bool:
        return True

    def _prepare_decode_scratch(self, batch: int, max_ctx: int):
        self._max_ctx = max_ctx

    def _forward(self, ids, pos, seq_ids, ctx_lens, prefill_shape=None, paged=None):
        """``paged`` as in the base class; without it every row is one token of the sequence ``seq_ids[row]``
        with ``ctx_lens[row]`` tokens including it (a decode step)."""
        if paged is not None:
            cu_q, kv_lens, table, max_q, slots, row_seq, max_kv = paged
        else:
            n = ids.numel()
            cu_q = torch.arange(n + 1, device=self.device, dtype=torch.int32)
            row_seq, slots, kv_lens, max_q, max_kv = cu_q[:n], seq_ids, ctx_lens, 1, self._max_ctx
            table = self.cache.block_table.index_select(0, slots)
        ctx = _Ctx([cu_q, kv_lens, slots, row_seq, pos], table, ids.numel(), kv_lens.numel(), max_q, max_kv)
        return self._run_layers(ids, pos, ctx)

    def _run_layers(self, ids, pos, ctx, trace=None):
        cfg, H = self.cfg, self.H
        d, eps = cfg.hidden_size, cfg.norm_eps
        x = self._new(ctx.rows, d, torch.float32)
        h = self._new(ctx.rows, _pad8(d))
        subs = []                                    # (layer, sublayer function, its norms)
        for L in self.layers:
            subs.append((L, self._parallel if L.spec.attention is not None else self._gla, L.norms))
            if L.spec.ff:
                subs.append((L, None, L.ff_norms))
        H.embed_pos_norm(ids, pos, self.embed_table, self.pos_table, cfg.embed_scale,
                         subs[0][2].pre if subs else self.final_norm, x, h, eps)
        for j, (L, fn, norms) in enumerate(subs):
            nxt = subs[j + 1][2].pre if j + 1 < len(subs) else self.final_norm
            if fn is None:
                H.sandwich_norm(self._feed_forward(L, h, ctx), None, None, None, norms.post, x, nxt, h, eps)
            else:
                y1, y2 = fn(L, h, ctx)
                H.sandwich_norm(y1, y2, L.left_norm, L.right_norm, norms.post, x, nxt, h, eps)
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
        return self._gemm(h, self.head, dtype=torch.float32, alpha=self.cfg.logit_scale)


class _HybridLayer:
    spec = norms = ff_norms = proj = a2 = g2 = out = left_out = right_out = left_norm = right_norm = rec = None
    gate_up = down = None
    rank = g_rank = att_index = 0

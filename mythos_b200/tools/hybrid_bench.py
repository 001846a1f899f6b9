"""Speed of layer-list models (Teganex, Lebedra, Dogozen or Zigivik layers at the sizes of a real model, random weights) beside
the dense transformer engine of equal width, depth and feed-forward (Lebedra, Dogozen: the dense layers', and the
experts of a token together about as wide), both with bf16 weights.

``run_models``: prefill and decode throughput of both engines. ``run_kernels``: every kernel of the new
design next to the like kernel of the dense model, with the fraction of its roofline (bytes over the
measured copy bandwidth or FLOPs over the measured bf16 GEMM rate). Timed with CUDA events on the launching
stream; L2 is flushed before every timed kernel, and the models' weights exceed it.
"""
from __future__ import annotations

import statistics

import torch

PAGE = 16


def _dense_config(width, layers, vocab, max_len):
    from ..models.config import TransformerConfig

    h = width // 128
    return TransformerConfig(vocab_size=vocab, hidden_size=width, num_layers=layers, num_heads=h, head_dim=128,
                             num_kv_heads=max(1, h // 8), ffn_hidden_size=width * 11 // 4 // 128 * 128, max_seq_len=max_len,
                             weight_format="bf16", embed_format="bf16")


def _engines(design, width, layers, vocab, batch, max_len):
    from ..infer.engine import InferenceEngine
    from ..infer.hybrid import HybridEngine
    from ..models import hybrid_config as hc

    kw = dict(seed=1, device="cuda", max_batch=batch, max_seq_len=max_len)
    make = {"teganex": hc.teganex_config, "lebedra": hc.lebedra_config, "dogozen": hc.dogozen_config, "zigivik": hc.zigivik_config}[design]
    yield design, HybridEngine.random(make(width, layers, vocab, max_len), **kw)
    yield "dense", InferenceEngine.random(_dense_config(width, layers, vocab, max_len), **kw)


def _event_ms(fn, iters: int, before=None) -> float:
    times = []
    for _ in range(iters):
        if before is not None:
            before()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
    return statistics.median(times)


def _prefill_ms(eng, batch, length, iters=4):
    g = torch.Generator().manual_seed(3)
    prompts = torch.randint(0, eng.cfg.vocab_size, (batch, length), generator=g, dtype=torch.int32)
    ms = []
    for i in range(iters + 3):
        seqs = [eng.cache.new_sequence() for _ in range(batch)]
        for s in seqs:
            eng.cache.reserve(s, length)
        eng.cache.sync_tables()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        eng._prefill_paged(seqs, [prompts[j] for j in range(batch)], [0] * batch)
        b.record()
        torch.cuda.synchronize()
        if i >= 3:
            ms.append(a.elapsed_time(b))
        for s in seqs:
            eng.release(s)
    return statistics.median(ms)


def run_models(design: str = "teganex", sizes=((2048, 8), (4096, 8)), vocab: int = 32000, prefill=((4, 2048), (1, 8192)),
               decode=((1, 1024), (16, 1024), (64, 1024)), new_tokens: int = 64) -> list[dict]:
    out = []
    for width, layers in sizes:
        max_len = max(max(n for _, n in prefill), max(n for _, n in decode) + new_tokens) + PAGE
        max_batch = max(max(b for b, _ in prefill), max(b for b, _ in decode))
        for name, eng in _engines(design, width, layers, vocab, max_batch, max_len):
            rec = {"model": name, "width": width, "layers": layers, "weight_mb": round(eng.weight_bytes() / 1e6), "prefill": [],
                   "decode": []}
            for b, n in prefill:
                ms = _prefill_ms(eng, b, n)
                rec["prefill"].append({"batch": b, "tokens": n, "ms": round(ms, 3), "tokens_per_s": round(b * n / ms * 1e3)})
            for b, n in decode:
                g = torch.Generator().manual_seed(4)
                p = torch.randint(0, vocab, (b, n), generator=g, dtype=torch.int32)
                best = min(eng.generate(p, max_new_tokens=new_tokens).stats.decode_s for _ in range(3))
                rec["decode"].append({"batch": b, "context": n, "ms_per_step": round(best / (new_tokens - 1) * 1e3, 4),
                                      "tokens_per_s": round(b * (new_tokens - 1) / best)})
            out.append(rec)
            del eng
            torch.cuda.empty_cache()
    return out


class _Kernels:
    """Times one call at a time and keeps (name, sizes, time, fraction of the roofline) rows."""

    def __init__(self, peaks: dict):
        self.hbm = float(peaks.get("hbm_gbs", 6650.0)) * 1e9
        self.tc = float(peaks.get("bf16_tflops", 1590.0)) * 1e12
        self.flush = torch.empty(64 << 20, device="cuda", dtype=torch.float32)
        self.rows = []

    def add(self, name, sizes, fn, nbytes=0.0, flops=0.0, like=None):
        for _ in range(3):
            fn()
        ms = _event_ms(fn, 10, before=lambda: self.flush.fill_(0.0))
        bound = max(nbytes / self.hbm, flops / self.tc) * 1e3
        self.rows.append({"kernel": name, "sizes": sizes, "us": round(ms * 1e3, 2), "bound_us": round(bound * 1e3, 2),
                          "fraction": round(bound / ms, 3), "like": like})


def _batch(lens, bases):
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    pos = torch.cat([torch.arange(b, b + n, dtype=torch.int32) for b, n in zip(bases, lens)]).cuda()
    row = torch.repeat_interleave(torch.arange(len(lens), dtype=torch.int32), torch.tensor(lens)).cuda()
    return [t(cu), t([b + n for b, n in zip(bases, lens)]), t(list(range(len(lens)))), row, pos]


def _recurrent_rows(K, H, st, kind, heads, dim, vdim, lens, decode):
    bf, n, slots = torch.bfloat16, sum(lens), len(lens)
    delta, taps = kind == "delta", 4 if kind == "delta" else 0
    cq, cv = heads * dim, heads * vdim
    off = {"q_off": 0, "k_off": cq, "v_off": 2 * cq, "b_off": 2 * cq + cv}
    spec = {"heads": heads, "kv_heads": heads, "dim": dim, "vdim": vdim, "taps": taps, "delta": int(delta), "unit_norm": int(delta),
            "decay_kind": int(delta), "gate_kind": int(delta), "q_scale": dim ** -0.5, "inv_tau": 1 / 16, "eps": 1e-6, **off}
    t = {"state": torch.zeros(slots, heads, vdim, dim), "z_bias": torch.full((cq,), -4.0 if delta else 3.0), "gamma": torch.ones(vdim)}
    if delta:
        t.update(a_log=torch.zeros(heads), conv_w=torch.randn(2 * cq + cv, taps), conv_state=torch.zeros(slots, taps - 1, 2 * cq + cv))
    rec = H.Recurrent(spec, {k: v.cuda() for k, v in t.items()})
    proj = torch.randn(n, 2 * cq + cv + heads, device="cuda").to(bf)
    z, gate = torch.randn(n, cq, device="cuda"), torch.randn(n, cv, device="cuda").to(bf)
    out, o = torch.empty(n, cv, device="cuda", dtype=bf), torch.empty(n, heads, vdim, device="cuda")
    sizes = f"{kind} {slots} x {n // slots}, {heads} heads, {dim} / {vdim}"
    io = n * (2 * cq + 2 * cv) * 2 + n * cq * 4 + n * cv * 2          # q, k, v, gate, decay in; gated output
    state = 2 * slots * heads * dim * vdim * 4
    if decode:
        b = _batch([1] * slots, [99] * slots)
        K.add("recurrent_decode", sizes, lambda: rec.decode(proj, z, gate, 0, 0, b, out), nbytes=io + state,
              like="paged decode attention (dense)")
        return
    b = _batch(lens, [0] * slots)
    scratch = torch.empty(rec.chunked_scratch(n, slots), device="cuda", dtype=torch.uint8)

    def fn():
        rec.scan_chunked(proj, z, b, scratch, o, st)
        rec.norm_gate(o, gate, out)

    K.add("chunked recurrence + norm + gate", sizes, fn, nbytes=io + state, like="paged prefill attention (dense)")


def _dense_attention_rows(K, H, C, st, rnd, h, kv):
    """Prefill and decode attention of the dense engine, for comparison."""
    bf, B, S = torch.bfloat16, 4, 2048
    pages = B * S // PAGE
    table = torch.randperm(pages, device="cuda").to(torch.int32).view(B, -1)
    kc, vc, q, o = rnd(pages, PAGE, kv, 128), rnd(pages, PAGE, kv, 128), rnd(B * S, h, 128), rnd(B * S, h, 128)
    b = _batch([S] * B, [0] * B)
    K.add("paged prefill attention (dense)", f"{B} x {S}, {h}/{kv} heads, 128",
          lambda: C.flash_attn_paged_prefill(q, kc, vc, table, b[0], b[1], o, S, 128 ** -0.5, st),
          flops=2.0 * B * h * (S * (S + 1) / 2) * 256)
    sms = torch.cuda.get_device_properties(0).multi_processor_count
    for NB, ctx in ((16, 4096), (64, 1024), (16, 1024), (1, 1024)):
        pages = NB * ctx // PAGE
        table = torch.randperm(pages, device="cuda").to(torch.int32).view(NB, -1)
        kc, vc, q, o = rnd(pages, PAGE, kv, 128), rnd(pages, PAGE, kv, 128), rnd(NB, h, 128), rnd(NB, h, 128)
        splits = max(1, min(32, (6 * sms + NB * kv - 1) // (NB * kv), (ctx + 255) // 256))
        b = _batch([1] * NB, [ctx - 1] * NB)
        scratch, cnt = torch.empty(NB * h * splits * 130, device="cuda"), torch.zeros(NB * kv, device="cuda", dtype=torch.int32)
        K.add("paged decode attention (dense)", f"{NB} x {ctx}, {h}/{kv} heads, 128",
              lambda: C.paged_attn_decode(q, kc, vc, table, b[1], o, scratch, cnt, splits, 128 ** -0.5, st),
              nbytes=4.0 * NB * ctx * kv * 128)


EXPERT_TOKENS = (1, 16, 64, 1024, 8192)


def _expert_rows(K, H, C, rnd, eng, L, T):
    """Routed experts of a layer for T tokens and the norms around them; gives two [T, width] activations."""
    from ..ops import functional as F

    e, d, bf, st = L.spec.mlp, eng.cfg.hidden_size, torch.bfloat16, eng._status
    route = (e.experts, e.top, e.groups, e.keep)
    i32 = dict(device="cuda", dtype=torch.int32)
    f, gen = e.ff, torch.Generator().manual_seed(5)
    pairs, tile = T * e.top, eng._expert_tile(T, e)
    z = torch.randn(T, e.experts, generator=gen).cuda()
    idx, slot, row = (torch.empty(T, e.top, **i32) for _ in range(3))
    wt, off, cnt = torch.empty(T, e.top, device="cuda"), torch.empty(e.experts, **i32), torch.empty(1, **i32)
    tiles = torch.empty(min(pairs, e.experts + pairs // tile), 3, **i32)
    plan = (idx, wt, slot, eng._expert_counts, off, tiles, cnt)
    x, hid, a, y = rnd(pairs, d), rnd(T, d), rnd(pairs, f), rnd(pairs, d)
    sizes = f"{T} tokens, {e.top} of {e.experts}, {d} x {f}"
    K.add("expert_select", sizes, lambda: H.expert_select(z, L.correction, route, tile, *plan, L.rule), nbytes=4.0 * T * e.experts,
          like="moe_route (training)")
    probs, psum, lg = torch.empty(T, e.experts, device="cuda"), torch.zeros(e.experts, device="cuda"), z.to(bf)
    cn = torch.zeros(e.experts, **i32)
    K.add("moe_route (training)", sizes, lambda: C.moe_route(lg, e.experts, probs, idx, slot, wt, cn, psum), nbytes=2.0 * T * e.experts)
    H.expert_select(z, L.correction, route, tile, *plan, L.rule)
    used = int((torch.bincount(idx.flatten().long(), minlength=e.experts) > 0).sum())
    K.add("expert_gather", sizes, lambda: H.expert_gather(hid, route, *plan, x, row), nbytes=2.0 * d * (T + pairs), like="rope (dense)")
    K.add("experts in (gate, up)", sizes, lambda: H.gemm_tiles(x, L.w_in, a, tiles, cnt, tile, f, f, L.act, st),
          nbytes=2.0 * (used * 2 * f * d + pairs * (d + f)), flops=4.0 * pairs * f * d, like="gemm (dense bf16)")
    K.add("experts out (down)", sizes, lambda: H.gemm_tiles(a, L.w_out, y, tiles, cnt, tile, 0, 0, L.act, st),
          nbytes=2.0 * (used * f * d + pairs * (d + f)), flops=2.0 * pairs * f * d, like="gemm (dense bf16)")
    for N, Kd in ((2 * f * e.top, d), (d, f * e.top)):         # the dense layer of the same width
        xx, ww, o1 = rnd(T, Kd), rnd(N, Kd), torch.empty(T, N, device="cuda", dtype=bf)
        K.add("gemm (dense bf16)", f"{T} x {N} x {Kd}", lambda: F.gemm(xx, ww, out=o1), nbytes=2.0 * (N * Kd + T * (N + Kd)),
              flops=2.0 * T * N * Kd)
    shared = rnd(T, d) if e.shared else None
    xs, w32, hh = torch.randn(T, d, device="cuda"), torch.ones(d, device="cuda"), rnd(T, d)
    nxt = w32 if eng.cfg.pre_norm else None
    K.add("expert_norm", f"{T} x {d}, {e.top} outputs", lambda: H.expert_norm(y, shared, row, wt, w32, xs, nxt, hh, 1e-6, 0.5),
          nbytes=T * d * (2.0 * e.top + 10 + 2 * (shared is not None)), like="rmsnorm + residual (dense)")
    K.add("norm + residual", f"{T} x {d}", lambda: H.sandwich_norm(hh, None, None, None, w32, xs, nxt, x[:T], 1e-6, 0.5),
          nbytes=T * d * 12.0, like="rmsnorm + residual (dense)")
    g, res = torch.ones(d, device="cuda", dtype=bf), rnd(T, d)
    K.add("rmsnorm + residual (dense)", f"{T} x {d}", lambda: F.rmsnorm(hh, g, 1e-6, res), nbytes=T * d * 8.0)
    return hid, hh


def _visible(S, w):
    """Query-key pairs of a sequence of S tokens."""
    return S * (S + 1) / 2 if not w or w >= S else w * (w + 1) / 2 + (S - w) * w


def run_zigivik_kernels(peaks: dict, width: int = 2048) -> list[dict]:
    """Window attention over latents, attention whose values are its keys, input convolution, PolyNorm and the stream."""
    from ..infer.hybrid import HybridEngine
    from ..models.hybrid_config import zigivik_config
    from ..ops import functional as F, native

    H, C, st = native.require_hybrid(), native.require(), native.status_word("cuda")
    K, bf, d = _Kernels(peaks), torch.bfloat16, width
    rnd = lambda *s: torch.randn(*s, device="cuda").to(bf)
    cfg = zigivik_config(width, 4, 32000)
    eng = HybridEngine.random(cfg, device="cuda", max_batch=64, max_seq_len=4096, kv_pages=64)
    L, full = eng.layers[0], eng.layers[3]
    m, a, ff, eps = L.spec.mixer, full.spec.mixer, L.spec.mlp.ff, cfg.norm_eps
    h, kv, r, W, win = m.heads, a.kv_heads, m.kv_rank, m.kv_rank + m.rot_dim, m.window
    dn, dv = m.dim, m.vdim
    _dense_attention_rows(K, H, C, st, rnd, h, kv)
    # ---- stream, convolution, PolyNorm
    for T in (1, 16, 64, 8192):
        b = _batch([1] * T, [99] * T) if T <= 64 else _batch([2048] * 4, [0] * 4)
        y, g, x = rnd(T, d), rnd(T, d), torch.randn(T, d, device="cuda")
        hid, bias, one = rnd(T, d), torch.zeros(d, device="cuda"), torch.ones(d, device="cuda")
        tail = (L.conv, b, g) if T <= 64 else None
        K.add("residual_norm" + (" + convolution" if tail else ""), f"{T} x {d}",
              lambda: H.residual_norm(y, bias, 0.7, x, one, hid, eps, tail), nbytes=T * d * (12.0 + (26 if tail else 0)),
              like="rmsnorm + residual (dense)")
        w16, res = torch.ones(d, device="cuda", dtype=bf), rnd(T, d)
        K.add("rmsnorm + residual (dense)", f"{T} x {d}", lambda: F.rmsnorm(hid, w16, 1e-6, res), nbytes=T * d * 8.0)
        if T > 64:
            K.add("input convolution", f"{T} x {d}", lambda: L.conv.run(hid, 0, b, False, g), nbytes=T * d * 4.0, like="rope (dense)")
        z, out = rnd(T, ff), rnd(T, L.out.shape[1])[:, L.mixer_cols:]
        K.add("poly_norm", f"{T} x {ff}", lambda: H.poly_norm(z, L.up_bias, L.poly, ff, out, eps), nbytes=T * ff * 4.0,
              like="rmsnorm + residual (dense)")
    # ---- attention whose values are its keys
    def pages(B, S):
        n = B * S // PAGE
        return torch.randperm(n, device="cuda").to(torch.int32).view(B, -1), rnd(n, PAGE, kv, 128), rnd(n, PAGE, kv, 128)

    for B, S in ((4, 2048), (1, 8192)):
        (table, kc, vc), b, n = pages(B, S), _batch([S] * B, [0] * B), B * S
        q, o, proj = rnd(n, h, 128), torch.empty(n, h * 128, device="cuda", dtype=bf), rnd(n, full.proj.N)
        K.add("attn_prep, pairs, keys as values", f"{n} tokens, {h}/{kv} heads, 128", lambda: full.att.prep(proj, b, table, q, kc, vc),
              nbytes=n * 128 * (4.0 * h + 6 * kv), like="rope (dense)")
        K.add("paged prefill attention, one in the denominator", f"{B} x {S}, {h}/{kv} heads, 128",
              lambda: full.att.prefill(q, kc, vc, b, table, None, o, S, st), flops=2.0 * B * h * _visible(S, 0) * 256,
              like="paged prefill attention (dense)")
    qkv, pos = rnd(8192, h + 2 * kv, 128), torch.arange(2048, device="cuda", dtype=torch.int32).repeat(4)
    K.add("rope (dense)", f"8192 tokens, {h}/{kv} heads, 128", lambda: C.rope(qkv[:, : h + kv], pos, 10000.0, False),
          nbytes=4.0 * 8192 * (h + kv) * 128)
    sms = torch.cuda.get_device_properties(0).multi_processor_count
    for NB, ctx in ((16, 4096), (64, 1024)):
        (table, kc, vc), b = pages(NB, ctx), _batch([1] * NB, [ctx - 1] * NB)
        q, o = rnd(NB, h, 128), torch.empty(NB, h * 128, device="cuda", dtype=bf)
        splits = max(1, min(32, (6 * sms + NB * kv - 1) // (NB * kv), (ctx + 255) // 256))
        scratch = torch.empty(full.att.decode_scratch(NB, splits), device="cuda")
        K.add("paged decode attention, one in the denominator", f"{NB} x {ctx}, {h}/{kv} heads, 128",
              lambda: full.att.decode(q, kc, vc, b, table, None, o, scratch, eng._counters, splits, st), nbytes=4.0 * NB * ctx * kv * 128,
              like="paged decode attention (dense)")
    # ---- window attention over latents
    def latents(B, S):
        return torch.randperm(B * S // PAGE, device="cuda").to(torch.int32).view(B, -1), rnd(B * S // PAGE, PAGE, 1, W)

    for B, S, past in ((4, 2048, 0), (1, 8192, 0), (4, 2048, 2048)):
        table, cache = latents(B, S + past)
        b, n, held = _batch([S] * B, [past] * B), B * S, S + min(past, win - 1)
        i32 = dict(device="cuda", dtype=torch.int32)
        cu = torch.arange(B + 1, **i32) * held
        first, keys = torch.full((B,), S + past - held, **i32), torch.full((B,), held, **i32)
        proj, qs, o = rnd(n, L.proj.N), rnd(n, L.low.N), torch.empty(n, h, dv, device="cuda", dtype=bf)
        lat, ex = torch.empty(B * held, W, device="cuda", dtype=bf), rnd(B * held, h * (dn + dv))
        q, k, v = qs[:, : h * dn].unflatten(1, (h, dn)), ex[:, : h * dn].unflatten(1, (h, dn)), ex[:, h * dn:].unflatten(1, (h, dv))
        gate, sizes = proj[:, L.proj.off["g"]:][:, : h * dv], f"{B} x {S}" + (f" behind {past}" if past else "")
        K.add("latent_prep, latents", sizes, lambda: L.lat.prep(proj, b, table, cache, queries=False),
              nbytes=4.0 * n * (W + m.q_rank), like="rope (dense)")
        K.add("latent_prep, queries", sizes, lambda: L.lat.prep(qs, b, table, cache, latents=False), nbytes=4.0 * n * h * m.rot_dim,
              like="rope (dense)")
        K.add("latent_gather", sizes, lambda: L.lat.gather(table, cache, cu, first, held, lat), nbytes=4.0 * B * held * W, like="rope (dense)")
        K.add(f"latent prefill attention, window {win}, gated", f"{sizes}, {h} heads, {dn} + {m.rot_dim} / {dv}",
              lambda: L.lat.attn_prefill(q, qs, k, v, lat, b, cu, keys, S, 16, gate, o, st),
              flops=2.0 * B * h * (_visible(S + past, win) - _visible(past, win)) * (dn + m.rot_dim + dv),
              nbytes=2.0 * n * h * (dn + m.rot_dim + 2 * dv), like="paged prefill attention (dense)")
    for NB, ctx in ((1, 4096), (16, 4096), (64, 4096)):
        table, cache = latents(NB, ctx)
        b, proj, qs = _batch([1] * NB, [ctx - 1] * NB), rnd(NB, L.proj.N), rnd(NB, L.low.N)
        ql, ol, out = rnd(NB, h, r), rnd(NB, h, r), rnd(NB, h, dv)
        q, gate = qs[:, : h * dn].unflatten(1, (h, dn)), proj[:, L.proj.off["g"]:][:, : h * dv]
        K.add("W_uk per head", f"{NB} tokens, {h} heads", lambda: H.gemm_heads(q, L.uk_t, ql, st),
              nbytes=2.0 * (L.uk_t.numel() + NB * h * (dn + r)), like="gemm_decode")
        splits = eng._latent_splits(NB, h, min(ctx, win + 64))
        sc = torch.empty(NB * h * splits * (r + 4), device="cuda")
        K.add(f"latent decode attention, window {win}", f"{NB} x {ctx}, {h} heads", lambda: L.lat.attn_decode(
            ql, qs, b[3], b[4], table, cache, ol, sc, splits, st),
            nbytes=2.0 * NB * (min(ctx, win) * W + h * (W + r)), flops=2.0 * NB * h * min(ctx, win) * (W + r),
            like=f"paged decode attention (dense), {NB} x {win}")
        K.add("W_uv per head, gated", f"{NB} tokens, {h} heads", lambda: H.gemm_heads(ol, L.uv, out, st, gate),
              nbytes=2.0 * (L.uv.numel() + NB * h * (2 * dv + r)), like="gemm_decode")
        x, w, y = rnd(NB, dn * 4), rnd(h * r // 4, dn * 4), rnd(NB, h * r // 4)
        K.add("gemm_decode", f"{NB} x {h * r // 4} x {dn * 4}", lambda: H.gemm_decode(x, w, y, 0, 0, 1.0, st),
              nbytes=2.0 * (w.numel() + x.numel() + y.numel()))
    # ---- products
    for T in (1, 16, 64, 8192):
        for name, ww in (("latent layer in", L.proj.weight), ("low-rank queries", L.low.weight), ("attention in", full.proj.weight),
                         ("feed-forward up", L.up), ("mixer and feed-forward out", L.out)):
            n_out, k_in = ww.shape
            xx, oo, sizes = rnd(T, k_in), torch.empty(T, n_out, device="cuda", dtype=bf), f"{T} x {n_out} x {k_in}"
            work = dict(nbytes=2.0 * (n_out * k_in + T * (k_in + n_out)), flops=2.0 * T * n_out * k_in)
            K.add(f"{name} (GEMM)", sizes, lambda: eng._gemm(xx, ww, out=oo), like="gemm (dense bf16)", **work)
            K.add("gemm (dense bf16)", sizes, lambda: F.gemm(xx, ww, out=oo), **work)
    native.check_status("cuda")
    return K.rows


def run_dogozen_kernels(peaks: dict, width: int = 2048) -> list[dict]:
    """Tempered and window attention (heads of 128), selective scan, routed and shared experts, soft-capped output."""
    from ..infer.hybrid import STEP_FUSE_ROWS, HybridEngine
    from ..models.hybrid_config import dogozen_config
    from ..ops import functional as F, native

    H, C, st = native.require_hybrid(), native.require(), native.status_word("cuda")
    K, bf, d = _Kernels(peaks), torch.bfloat16, width
    rnd = lambda *s: torch.randn(*s, device="cuda").to(bf)
    cfg = dogozen_config(width, 2, 32000)
    eng = HybridEngine.random(cfg, device="cuda", max_batch=64, max_seq_len=4096, kv_pages=64)
    full, par = eng.layers
    h, kv, r = full.spec.mixer.heads, full.spec.mixer.kv_heads, par.spec.mixer.right
    win, sms = par.spec.mixer.left.window, torch.cuda.get_device_properties(0).multi_processor_count
    _dense_attention_rows(K, H, C, st, rnd, h, kv)

    def pages(B, S):
        n = B * S // PAGE
        return torch.randperm(n, device="cuda").to(torch.int32).view(B, -1), rnd(n, PAGE, kv, 128), rnd(n, PAGE, kv, 128)

    # ---- attention
    kinds = (("tempered, gated", full, 0), (f"window {win}, sink", par, win))
    for B, S in ((4, 2048), (1, 8192)):
        (table, kc, vc), b, n = pages(B, S), _batch([S] * B, [0] * B), B * S
        q, o = rnd(n, h, 128), torch.empty(n, h * 128, device="cuda", dtype=bf)
        for name, L, w in kinds:
            proj = rnd(n, L.proj.N)
            gate = proj[:, L.proj.off["g"]:][:, : h * 128] if "g" in L.proj.off else None
            K.add(f"attn_prep, {name}", f"{n} tokens, {h}/{kv} heads, 128", lambda: L.att.prep(proj, b, table, q, kc, vc),
                  nbytes=4.0 * n * (h + 2 * kv) * 128, like="rope (dense)")
            K.add(f"paged prefill attention, {name}", f"{B} x {S}, {h}/{kv} heads, 128",
                  lambda: L.att.prefill(q, kc, vc, b, table, gate, o, S, st), flops=2.0 * B * h * _visible(S, w) * 256,
                  nbytes=n * (h * 128 * (4.0 + 2 * (gate is not None)) + 512 * kv), like="paged prefill attention (dense)")
    qkv, pos = rnd(8192, h + 2 * kv, 128), torch.arange(2048, device="cuda", dtype=torch.int32).repeat(4)
    K.add("rope (dense)", f"8192 tokens, {h}/{kv} heads, 128", lambda: C.rope(qkv[:, : h + kv], pos, 10000.0, False),
          nbytes=4.0 * 8192 * (h + kv) * 128)
    for NB, ctx in ((16, 4096), (64, 1024), (64, 4096)):
        (table, kc, vc), b = pages(NB, ctx), _batch([1] * NB, [ctx - 1] * NB)
        q, o = rnd(NB, h, 128), torch.empty(NB, h * 128, device="cuda", dtype=bf)
        for name, L, w in kinds:
            proj, keys = rnd(NB, L.proj.N), min(ctx, w or ctx)
            gate = proj[:, L.proj.off["g"]:][:, : h * 128] if "g" in L.proj.off else None
            splits = max(1, min(32, (6 * sms + NB * kv - 1) // (NB * kv), (keys + (PAGE if w else 0) + 255) // 256))
            scratch = torch.empty(L.att.decode_scratch(NB, splits), device="cuda")
            K.add(f"paged decode attention, {name}", f"{NB} x {ctx}, {h}/{kv} heads, 128",
                  lambda: L.att.decode(q, kc, vc, b, table, gate, o, scratch, eng._counters, splits, st), nbytes=4.0 * NB * keys * kv * 128,
                  like="paged decode attention (dense)")
    # ---- selective scan
    c, ns, sel, N = r.inner, r.state, par.sel, par.proj.N
    for B, S in ((16, 512), (4, 2048), (1, 8192)):
        n, b = B * S, _batch([S] * B, [0] * B)
        proj, x, low, out = rnd(n, N), rnd(n, c), rnd(n, par.x_maps.N), torch.empty(n, c, device="cuda", dtype=bf)
        dt, sizes = torch.randn(n, c, device="cuda") - 3.0, f"{B} x {S}, {c} channels, {ns} state values"
        scratch = torch.empty(sel.scratch_floats(B, n, S), device="cuda")
        K.add("selective_conv", sizes, lambda: par.conv.run(proj, par.proj.off["rx"], b, False, x), nbytes=4.0 * n * c, like="rope (dense)")
        K.add("selective_scan", sizes, lambda: sel.scan(proj, x, low, dt, b, S, scratch, out, st),
              nbytes=n * (c * 10.0 + 4 * ns) + 8.0 * B * c * ns, like="chunked recurrence + norm + gate")
        _recurrent_rows(K, H, st, "delta", h, 128, 128, [S] * B, False)
        _recurrent_rows(K, H, st, "gla", h, 64, 128, [S] * B, False)
    for T in (1, 16, 64):
        b = _batch([1] * T, [99] * T)
        proj, x, low, out = rnd(T, N), rnd(T, c), rnd(T, par.x_maps.N), torch.empty(T, c, device="cuda", dtype=bf)
        dt = torch.randn(T, c, device="cuda") if T > STEP_FUSE_ROWS else None
        sizes = f"{T} tokens, {c} channels, {ns} state values"
        K.add("selective_conv, one token", sizes, lambda: par.conv.run(proj, par.proj.off["rx"], b, True, x), nbytes=T * c * (4.0 + 24), like="recurrent_decode")
        K.add("selective_step", sizes, lambda: sel.step(proj, x, low, dt, b, out),
              nbytes=T * c * (8.0 * ns + 6 + 4 * (dt is not None)) + 2.0 * c * r.dt_rank * (dt is None), like="recurrent_decode")
        _recurrent_rows(K, H, st, "delta", h, 128, 128, [1] * T, True)
        _recurrent_rows(K, H, st, "gla", h, 64, 128, [1] * T, True)
    for T in EXPERT_TOKENS:
        proj, x, low = rnd(T, N), rnd(T, c), rnd(T, par.x_maps.N)
        dt, y, z = torch.empty(T, c, device="cuda"), rnd(T, par.out.shape[1]), rnd(T, d)
        R = par.w_dt.shape[1]
        for name, xx, ww, oo, like in (
                ("mixer in", z, par.proj.weight, proj, "gemm (dense bf16)"), ("mixer out, both mixers", y, par.out, z, "gemm (dense bf16)"),
                ("maps of the scan", x, par.x_maps.weight, low, "gemm (dense bf16), narrow"),
                ("step sizes", low[:, :R], par.w_dt, dt, "gemm (dense bf16), narrow")):
            n_out, k_in = ww.shape
            nb = 2.0 * (n_out * k_in + T * (k_in + n_out * oo.element_size() / 2))
            K.add(f"{name} (GEMM)", f"{T} x {n_out} x {k_in}", lambda: eng._gemm(xx, ww, out=oo), nbytes=nb, flops=2.0 * T * n_out * k_in,
                  like=like)
            x2, o2 = rnd(T, k_in), torch.empty(T, n_out, device="cuda", dtype=bf)
            K.add(like, f"{T} x {n_out} x {k_in}", lambda: F.gemm(x2, ww, out=o2), nbytes=2.0 * (n_out * k_in + T * (k_in + n_out)),
                  flops=2.0 * T * n_out * k_in)
    # ---- experts, output
    for T in EXPERT_TOKENS:
        hid, _ = _expert_rows(K, H, C, rnd, eng, par, T)
    for T in (1, 64):
        x, lg, lb = rnd(T, d), torch.empty(T, 32000, device="cuda"), torch.empty(T, 32000, device="cuda", dtype=bf)
        nb = 2.0 * (32000 * d + T * (d + 64000))
        K.add("soft-capped output (GEMM)", f"{T} x 32000 x {d}", lambda: eng._gemm(x, eng.head, out=lg, cap=50.0), nbytes=nb,
              flops=2.0 * T * 32000 * d, like="gemm (dense bf16)")
        K.add("gemm (dense bf16)", f"{T} x 32000 x {d}", lambda: F.gemm(x, eng.head, out=lb), nbytes=nb, flops=2.0 * T * 32000 * d)
    native.check_status("cuda")
    return K.rows


def run_lebedra_kernels(peaks: dict, width: int = 2048) -> list[dict]:
    """Latent attention (latents of 512, heads of 128 + 64 rotated), routed experts and the norms around them."""
    from ..infer.hybrid import HybridEngine
    from ..models.hybrid_config import lebedra_config
    from ..ops import functional as F, native

    H, C, st = native.require_hybrid(), native.require(), native.status_word("cuda")
    K, bf, d = _Kernels(peaks), torch.bfloat16, width
    rnd = lambda *s: torch.randn(*s, device="cuda").to(bf)
    cfg = lebedra_config(width, 2, 1024)
    eng = HybridEngine.random(cfg, device="cuda", max_batch=64, max_seq_len=4096, kv_pages=64)
    L, m, e = eng.layers[1], cfg.layers[1].mixer, cfg.layers[1].mlp
    h, r, W = m.heads, m.kv_rank, m.kv_rank + m.rot_dim
    _dense_attention_rows(K, H, C, st, rnd, h, max(1, h // 8))
    # ---- attention
    def pages(B, S):
        return torch.randperm(B * S // PAGE, device="cuda").to(torch.int32).view(B, -1), rnd(B * S // PAGE, PAGE, 1, W)

    for B, S in ((4, 2048), (1, 8192)):
        table, cache = pages(B, S)
        b, n, zero = _batch([S] * B, [0] * B), B * S, torch.zeros(B, device="cuda", dtype=torch.int32)
        proj, o = rnd(n, L.proj.N), torch.empty(n, h, m.vdim, device="cuda", dtype=bf)
        lat, kv = torch.empty(n, W, device="cuda", dtype=bf), rnd(n, h * (m.dim + m.vdim))
        q, k, v = (t.unflatten(1, (h, 128)) for t in (proj[:, : h * m.dim], kv[:, : h * m.dim], kv[:, h * m.dim:]))
        K.add("latent_prep", f"{n} tokens, {h} heads", lambda: L.lat.prep(proj, b, table, cache),
              nbytes=2.0 * n * (2 * h * m.rot_dim + 2 * W), like="rope (dense)")
        K.add("latent_gather", f"{n} tokens", lambda: L.lat.gather(table, cache, b[0], zero, S, lat), nbytes=4.0 * n * W, like="rope (dense)")
        K.add("expand latents (GEMM)", f"{n} x {L.expand.shape[0]} x {r}", lambda: H.gemm_nt(lat[:, :r], L.expand, kv, 1.0, st),
              flops=2.0 * n * L.expand.shape[0] * r, like="gemm (dense bf16)")
        K.add("latent prefill attention", f"{B} x {S}, {h} heads, 128 + 64 / 128",
              lambda: L.lat.attn_prefill(q, proj, k, v, lat, b, b[0], b[1], S, 16, None, o, st),
              flops=2.0 * B * h * (S * (S + 1) / 2) * (m.dim + m.rot_dim + m.vdim), like="paged prefill attention (dense)")
    qkv, pos = rnd(8192, h + 2, 128), torch.arange(2048, device="cuda", dtype=torch.int32).repeat(4)
    K.add("rope (dense)", f"8192 tokens, {h} heads, 128", lambda: C.rope(qkv[:, :h], pos, 10000.0, False), nbytes=4.0 * 8192 * h * 128)
    for NB, ctx in ((1, 4096), (16, 4096), (64, 1024)):
        table, cache = pages(NB, ctx)
        b, proj = _batch([1] * NB, [ctx - 1] * NB), rnd(NB, L.proj.N)
        ql, ol, out = rnd(NB, h, r), rnd(NB, h, r), rnd(NB, h, m.vdim)
        q = proj[:, : h * m.dim].unflatten(1, (h, m.dim))
        K.add("W_uk per head", f"{NB} tokens, {h} heads", lambda: H.gemm_heads(q, L.uk_t, ql, st),
              nbytes=2.0 * (L.uk_t.numel() + NB * h * (m.dim + r)), like="gemm_decode")
        splits = eng._latent_splits(NB, h, ctx)
        sc = torch.empty(NB * h * splits * (r + 4), device="cuda")
        K.add("latent decode attention", f"{NB} x {ctx}, {h} heads", lambda: L.lat.attn_decode(
            ql, proj, b[3], b[4], table, cache, ol, sc, splits, st),
            nbytes=2.0 * NB * (ctx * W + h * (W + r)), flops=2.0 * NB * h * ctx * (W + r), like="paged decode attention (dense)")
        K.add("W_uv per head", f"{NB} tokens, {h} heads", lambda: H.gemm_heads(ol, L.uv, out, st),
              nbytes=2.0 * (L.uv.numel() + NB * h * (m.vdim + r)), like="gemm_decode")
        N = h * r
        x, w, y = rnd(NB, m.dim * 4), rnd(N // 4, m.dim * 4), rnd(NB, N // 4)
        K.add("gemm_decode", f"{NB} x {N // 4} x {m.dim * 4}", lambda: H.gemm_decode(x, w, y, 0, 0, 1.0, st),
              nbytes=2.0 * (w.numel() + x.numel() + y.numel()))
    # ---- experts
    for T in EXPERT_TOKENS:
        hid, hh = _expert_rows(K, H, C, rnd, eng, L, T)
        # ---- token side and router
        n, ids = cfg.token_side, torch.zeros(T, device="cuda", dtype=torch.int32)
        sg = torch.empty(T, n, device="cuda", dtype=bf)
        K.add("side gate", f"{T} x {n} x {d}", lambda: H.gemm_decode(hid, L.side_gate, sg, 0, 0, 1.0, st, (0, 0.0, 0.0), L.side_embed, ids),
              nbytes=2.0 * (n * d + T * (d + 2 * n)), flops=2.0 * T * n * d, like="gemm (dense bf16), narrow")
        K.add("gemm (dense bf16), narrow", f"{T} x {n} x {d}", lambda: F.gemm(hid, L.side_gate, out=sg), nbytes=2.0 * (n * d + T * (d + n)),
              flops=2.0 * T * n * d)
        K.add("side projection", f"{T} x {d} x {n}", lambda: eng._gemm(sg, L.side_proj, out=hh), nbytes=2.0 * (n * d + T * (d + n)),
              flops=2.0 * T * n * d, like="gemm (dense bf16), narrow")
        zz = torch.empty(T, e.experts, device="cuda")
        K.add("router", f"{T} x {e.experts} x {d}", lambda: eng._gemm(hid, L.router, out=zz),
              nbytes=2.0 * (e.experts * d + T * (d + 2 * e.experts)), flops=2.0 * T * e.experts * d, like="gemm (dense bf16), narrow")
    native.check_status("cuda")
    return K.rows


def run_kernels(peaks: dict, width: int = 2048, design: str = "teganex") -> list[dict]:
    if design == "lebedra":
        return run_lebedra_kernels(peaks, width)
    if design == "dogozen":
        return run_dogozen_kernels(peaks, width)
    if design == "zigivik":
        return run_zigivik_kernels(peaks, width)
    from ..ops import functional as F, native

    H, C, st = native.require_hybrid(), native.require(), native.status_word("cuda")
    K, bf, d = _Kernels(peaks), torch.bfloat16, width
    rnd = lambda *s: torch.randn(*s, device="cuda").to(bf)
    h, ff = width // 128, width * 11 // 4 // 128 * 128
    # ---- norms
    for T in (64, 8192):
        y1, y2, out = rnd(T, d), rnd(T, d), rnd(T, d)
        x, w = torch.randn(T, d, device="cuda"), torch.ones(d, device="cuda")
        K.add("sandwich_norm", f"{T} x {d}", lambda: H.sandwich_norm(y1, None, None, None, w, x, w, out, 1e-6), nbytes=T * d * 12,
              like="rmsnorm + residual (dense)")
        K.add("sandwich_norm, two mixers", f"{T} x {d}", lambda: H.sandwich_norm(y1, y2, w, w, w, x, w, out, 1e-6), nbytes=T * d * 14,
              like="rmsnorm + residual (dense)")
        g = torch.ones(d, device="cuda", dtype=bf)
        K.add("rmsnorm + residual (dense)", f"{T} x {d}", lambda: F.rmsnorm(y1, g, 1e-6, y2), nbytes=T * d * 8)
    # ---- few-token GEMM
    for T in (1, 16, 64):
        for name, N, Kd in (("mixer in", 8 * d, d), ("mixer out", d, d), ("down", d, ff)):
            xx, ww = rnd(T, Kd), rnd(N, Kd)
            o1 = torch.empty(T, N, device="cuda", dtype=bf)
            nb = 2.0 * (N * Kd + T * (N + Kd))
            K.add(f"gemm_decode, {name}", f"{T} x {N} x {Kd}", lambda: H.gemm_decode(xx, ww, o1, 0, 0, 1.0, st), nbytes=nb,
                  flops=2.0 * T * N * Kd, like="gemm (dense bf16)")
            K.add("gemm (dense bf16)", f"{T} x {N} x {Kd}", lambda: F.gemm(xx, ww, out=o1), nbytes=nb, flops=2.0 * T * N * Kd)
    # ---- attention
    B, S = 4, 2048
    pages = B * S // PAGE
    table = torch.randperm(pages, device="cuda").to(torch.int32).view(B, -1)
    kv = max(1, h // 8)
    for dk, dv in ((128, 128), (64, 128)):
        kc, vc = rnd(pages, PAGE, kv, dk), rnd(pages, PAGE, kv, dv)
        b = _batch([S] * B, [0] * B)
        q, gate, o = rnd(B * S, h, dk), rnd(B * S, h), torch.empty(B * S, h * dv, device="cuda", dtype=bf)
        proj, ones = rnd(B * S, h * dk + kv * (dk + dv)), torch.ones(dk, device="cuda")
        att = H.Attention({"heads": h, "kv_heads": kv, "dk": dk, "dv": dv, "k_off": h * dk, "v_off": (h + kv) * dk, "norm_dim": dk,
                           "scale": dk ** -0.5}, {"q_gamma": ones, "k_gamma": ones})
        fl = 2.0 * B * h * (S * (S + 1) / 2) * (dk + dv)
        K.add("gated paged prefill attention", f"{B} x {S}, {h}/{kv} heads, {dk} / {dv}",
              lambda: att.prefill(q, kc, vc, b, table, gate, o, S, st), flops=fl, like="paged prefill attention (dense)")
        if dk == dv:
            o3 = o.view(B * S, h, dv)
            K.add("paged prefill attention (dense)", f"{B} x {S}, {h}/{kv} heads, {dk}",
                  lambda: C.flash_attn_paged_prefill(q, kc, vc, table, b[0], b[1], o3, S, dk ** -0.5, st), flops=fl)
        K.add("attn_prep, norm", f"{B * S} tokens, {h}/{kv} heads, {dk} / {dv}", lambda: att.prep(proj, b, table, q, kc, vc),
              nbytes=4.0 * B * S * (h * dk + kv * (dk + dv)), like="rope (dense)")
    qkv, pos = rnd(B * S, h + 2 * kv, 128), torch.arange(S, device="cuda", dtype=torch.int32).repeat(B)
    K.add("rope (dense)", f"{B * S} tokens, {h}/{kv} heads, 128", lambda: C.rope(qkv[:, : h + kv], pos, 10000.0, False),
          nbytes=4.0 * B * S * (h + kv) * 128)
    for NB, ctx in ((16, 4096), (64, 1024)):
        pages = NB * ctx // PAGE
        table = torch.randperm(pages, device="cuda").to(torch.int32).view(NB, -1)
        sms = torch.cuda.get_device_properties(0).multi_processor_count
        splits = max(1, min(32, (6 * sms + NB * kv - 1) // (NB * kv), (ctx + 255) // 256))
        for dk, dv in ((128, 128), (64, 128)):
            kc, vc = rnd(pages, PAGE, kv, dk), rnd(pages, PAGE, kv, dv)
            q, gate, o = rnd(NB, h, dk), rnd(NB, h), torch.empty(NB, h * dv, device="cuda", dtype=bf)
            b = _batch([1] * NB, [ctx - 1] * NB)
            att = H.Attention({"heads": h, "kv_heads": kv, "dk": dk, "dv": dv, "scale": dk ** -0.5}, {})
            scratch, cnt = torch.empty(NB * h * splits * (dv + 2), device="cuda"), torch.zeros(NB * kv, device="cuda", dtype=torch.int32)
            nb = 2.0 * NB * ctx * kv * (dk + dv)
            K.add("gated paged decode attention", f"{NB} x {ctx}, {h}/{kv} heads, {dk} / {dv}",
                  lambda: att.decode(q, kc, vc, b, table, gate, o, scratch, cnt, splits, st), nbytes=nb,
                  like="paged decode attention (dense)")
            if dk == dv:
                o3 = o.view(NB, h, dv)
                K.add("paged decode attention (dense)", f"{NB} x {ctx}, {h}/{kv} heads, {dk}",
                      lambda: C.paged_attn_decode(q, kc, vc, table, b[1], o3, scratch, cnt, splits, dk ** -0.5, st), nbytes=nb)
    # ---- recurrences
    for lens in ([2048] * 4, [8192], [512] * 16):
        _recurrent_rows(K, H, st, "delta", h, 128, 128, lens, False)
        _recurrent_rows(K, H, st, "gla", h, 64, 128, lens, False)
    for NB in (1, 16, 64):
        _recurrent_rows(K, H, st, "delta", h, 128, 128, [1] * NB, True)
        _recurrent_rows(K, H, st, "gla", h, 64, 128, [1] * NB, True)
    native.check_status("cuda")
    return K.rows


def main(argv=None) -> int:
    import argparse
    import json
    import os

    ap = argparse.ArgumentParser(description=__doc__)
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--models", action="store_true")
    ap.add_argument("--width", type=int, default=2048)
    ap.add_argument("--design", default="teganex", choices=["teganex", "lebedra", "dogozen", "zigivik"])
    a = ap.parse_args(argv)
    peaks = {}
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            peaks = json.load(f)
    if a.kernels or not a.models:
        for r in run_kernels(peaks, a.width, a.design):
            print(json.dumps(r), flush=True)
    if a.models or not a.kernels:
        for r in run_models(a.design):
            print(json.dumps(r), flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())

"""Speed of layer-list models (Teganex layers at the sizes of a real model, random weights) beside the
dense transformer engine of equal width, depth and feed-forward, both with bf16 weights.

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


def _engines(width, layers, vocab, batch, max_len):
    from ..infer.engine import InferenceEngine
    from ..infer.hybrid import HybridEngine
    from ..models.hybrid_config import teganex_config

    kw = dict(seed=1, device="cuda", max_batch=batch, max_seq_len=max_len)
    yield "teganex", HybridEngine.random(teganex_config(width, layers, vocab, max_len), **kw)
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


def run_models(sizes=((2048, 8), (4096, 8)), vocab: int = 32000, prefill=((4, 2048), (1, 8192)),
               decode=((1, 1024), (16, 1024), (64, 1024)), new_tokens: int = 64) -> list[dict]:
    out = []
    for width, layers in sizes:
        max_len = max(max(n for _, n in prefill), max(n for _, n in decode) + new_tokens) + PAGE
        max_batch = max(max(b for b, _ in prefill), max(b for b, _ in decode))
        for name, eng in _engines(width, layers, vocab, max_batch, max_len):
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


def run_kernels(peaks: dict, width: int = 2048) -> list[dict]:
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
        fl = 2.0 * B * h * (S * (S + 1) / 2) * (dk + dv)
        K.add("gated paged prefill attention", f"{B} x {S}, {h}/{kv} heads, {dk} / {dv}",
              lambda: H.paged_attn_prefill(q, kc, vc, b, table, gate, o, S, dk ** -0.5, st), flops=fl, like="paged prefill attention (dense)")
        if dk == dv:
            o3 = o.view(B * S, h, dv)
            K.add("paged prefill attention (dense)", f"{B} x {S}, {h}/{kv} heads, {dk}",
                  lambda: C.flash_attn_paged_prefill(q, kc, vc, table, b[0], b[1], o3, S, dk ** -0.5, st), flops=fl)
        proj, ones = rnd(B * S, h * dk + kv * (dk + dv)), torch.ones(dk, device="cuda")
        K.add("qk_norm_append", f"{B * S} tokens, {h}/{kv} heads, {dk} / {dv}",
              lambda: H.qk_norm_append(proj, 0, h * dk, (h + kv) * dk, ones, ones, b, table, q, kc, vc, 1e-6),
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
            scratch, cnt = torch.empty(NB * h * splits * (dv + 2), device="cuda"), torch.zeros(NB * kv, device="cuda", dtype=torch.int32)
            nb = 2.0 * NB * ctx * kv * (dk + dv)
            K.add("gated paged decode attention", f"{NB} x {ctx}, {h}/{kv} heads, {dk} / {dv}",
                  lambda: H.paged_attn_decode(q, kc, vc, b, table, gate, o, scratch, cnt, splits, dk ** -0.5, st), nbytes=nb,
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
    a = ap.parse_args(argv)
    peaks = {}
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            peaks = json.load(f)
    if a.kernels or not a.models:
        for r in run_kernels(peaks, a.width):
            print(json.dumps(r), flush=True)
    if a.models or not a.kernels:
        for r in run_models():
            print(json.dumps(r), flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())

"""Layer-list models on the GPU against the plain implementation in ``hybrid_oracle``: each kernel alone,
then the engine (prompts, portions, decoding, batches, reuse of pages and slots, generation)."""
import json
import os
import subprocess
import sys

import pytest
import torch

import hybrid_oracle as oracle
import hybrid_util as hu

pytestmark = pytest.mark.gpu

TOL = {"float32": 5e-5, "bfloat16": 6e-2}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def H():
    from mythos_b200.ops import native

    return native.require_hybrid()


def status():
    from mythos_b200.ops import native

    return native.status_word("cuda")


def engine(cfg, dtype="bfloat16", seed=0, w=None, **kw):
    from mythos_b200.infer.engine import InferenceEngine

    kw.setdefault("max_batch", 4)
    kw.setdefault("max_seq_len", 640)
    return InferenceEngine.from_model(hu.model(cfg, seed, w=w), device="cuda", dtype=dtype, **kw)


def ragged(lens, bases=None, slots=None):
    """(cu_q, kv_lens, slots, row_seq, pos) of a batch."""
    n = len(lens)
    bases = bases or [0] * n
    cu = [0]
    for k in lens:
        cu.append(cu[-1] + k)
    i = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    pos = [b + j for b, k in zip(bases, lens) for j in range(k)]
    row = [s for s, k in enumerate(lens) for _ in range(k)]
    return [i(cu), i([b + k for b, k in zip(bases, lens)]), i(slots or list(range(n))), i(row), i(pos)]


def close(a, b, tol):
    assert a.shape == b.shape
    a, b = a.double().cpu(), b.double().cpu()
    assert torch.isfinite(a).all()
    err = float((a - b).abs().max()) / max(1e-9, float(b.abs().max()))
    assert err <= tol, f"{err} > {tol}"


class Truth:
    """The oracle's logits and streams for one sequence."""

    def __init__(self, cfg, w, toks):
        self.layers, self.routed = [], cfg["architecture"] in ("Lebedra", "Dogozen")
        self.logits = oracle.forward(cfg, w, toks, trace=self.layers)

    def agrees(self, got, dtype, rows=slice(None), layer=None):
        """Every row within the tolerance; in bf16, up to one row in thirty may be a small output whose rounding the norm
        behind it enlarges (norms on outputs only), or a close call of a router."""
        want = self.logits if layer is None else self.layers[layer]
        e = hu.row_errors(got, want[rows], want)
        over = int((e >= TOL[dtype]).sum())
        return bool(torch.isfinite(got).all()) and over <= (max(1, e.numel() // 30) if self.routed and dtype == "bfloat16" else 0)


def model_weights(cfg, seed, dtype):
    return hu.weights(cfg, seed, sure_routes=dtype == "bfloat16")


# ------------------------------------------------------------------------------- single kernels
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,dim,two", [(3, 100, False), (5, 333, True), (2, 2048, True), (7, 64, False)])
def test_sandwich_norm(dtype, rows, dim, two):
    torch.manual_seed(dim)
    ld = (dim + 7) // 8 * 8
    y1, y2 = (torch.randn(rows, dim, device="cuda").to(dtype) * 3 for _ in range(2))
    w1, w2, wp, wn = (1 + 0.3 * torch.randn(dim, device="cuda") for _ in range(4))
    x = torch.randn(rows, dim, device="cuda")
    x0 = x.double().cpu()
    h = torch.full((rows, ld), float("nan"), device="cuda", dtype=dtype)
    H().sandwich_norm(y1, y2 if two else None, w1 if two else None, w2 if two else None, wp, x, wn, h, 1e-3)
    d = lambda t: t.double().cpu()
    y = d(y1)
    if two:
        y = 0.5 * (oracle.rms_norm(d(y1), d(w1), 1e-3) + oracle.rms_norm(d(y2), d(w2), 1e-3))
    want = x0 + oracle.rms_norm(y, d(wp), 1e-3)
    close(x, want, 1e-6)
    close(h[:, :dim], oracle.rms_norm(want, d(wn), 1e-3), 1e-6 if dtype == torch.float32 else 1e-2)
    assert float(h[:, dim:].float().abs().sum()) == 0.0


def test_embedding_with_positions_and_first_norm():
    torch.manual_seed(0)
    V, P, dim = 50, 40, 76
    emb, pos = torch.randn(V, dim, device="cuda"), torch.randn(P, dim, device="cuda")
    ids = torch.randint(0, V, (9,), device="cuda", dtype=torch.int32)
    at = torch.tensor([0, 1, 2, 39, 5, 6, 0, 1, 20], device="cuda", dtype=torch.int32)
    g = torch.rand(dim, device="cuda") + 0.5
    x, h = torch.empty(9, dim, device="cuda"), torch.empty(9, 80, device="cuda")
    H().embed_pos_norm(ids, at, emb, pos, 0.25, g, x, h, 1e-5)
    want = emb[ids.long()].double() * 0.25 + pos[at.long()].double()
    close(x, want, 1e-6)
    close(h[:, :dim], oracle.rms_norm(want.cpu(), g.double().cpu(), 1e-5), 1e-6)


@pytest.mark.parametrize("M,N,K", [(1, 100, 72), (5, 257, 64), (64, 1024, 2048), (17, 128, 200), (128, 384, 512), (130, 96, 1000)])
def test_few_token_gemm(M, N, K):
    torch.manual_seed(M)
    x, w = (torch.randn(r, K, device="cuda").to(torch.bfloat16) for r in (M, N))
    ref = x.double() @ w.double().t()
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
        out = torch.full((M, N), float("nan"), device="cuda", dtype=dt)
        H().gemm_decode(x, w, out, 0, 0, 0.5, status())
        close(out, 0.5 * ref, tol)
    f = N // 16 * 8                                        # gate rows [0, f), up rows from an offset past them
    off = f + 8 if f + 8 + f <= N else f
    out = torch.full((M, f), float("nan"), device="cuda", dtype=torch.bfloat16)
    H().gemm_decode(x / 8, w, out, f, off, 1.0, status())
    close(out, oracle.silu(ref[:, :f] / 8) * ref[:, off:off + f] / 8, 1e-2)


def test_gemm_fp32_is_true_32_bit():
    torch.manual_seed(1)
    a, b = torch.randn(70, 150, device="cuda"), torch.randn(91, 150, device="cuda")
    out = torch.empty(70, 91, device="cuda")
    H().gemm_nt(a, b, out, 1.0, None)
    close(out, a.double() @ b.double().t(), 1e-6)


def _attention_case(dtype, heads, kv, dk, dv, lens, bases, seed=0):
    """Paged keys and values with everything before the new tokens already in shuffled pages, and the
    projections of the new tokens."""
    g = torch.Generator().manual_seed(seed)
    n, page = len(lens), 16
    total = [b + k for b, k in zip(bases, lens)]
    need = [(t + page - 1) // page for t in total]
    order = torch.randperm(sum(need) + 3, generator=g).tolist()
    table = torch.full((n, max(need) + 1), -1, dtype=torch.int32)
    kc = torch.randn(len(order), page, kv, dk, generator=g)   # unused pages hold other finite values
    vc = torch.randn(len(order), page, kv, dv, generator=g)
    for s in range(n):
        for i in range(need[s]):
            table[s, i] = order.pop()
    rows = sum(lens)
    off = [0, (heads * dk + 7) // 8 * 8]
    off.append(off[1] + (kv * dk + 7) // 8 * 8)
    ld = off[2] + (kv * dv + 7) // 8 * 8
    proj = torch.randn(rows, ld, generator=g)
    gate = torch.randn(rows, (heads + 7) // 8 * 8, generator=g)
    c = lambda t: t.to("cuda", dtype)
    return dict(table=table.cuda(), kc=c(kc), vc=c(vc), proj=c(proj), off=off, gate=c(gate), lens=lens, bases=bases,
                heads=heads, kv=kv, dk=dk, dv=dv, batch=ragged(lens, bases), total=total)


def _run_attention(case, kernel, gamma_q, gamma_k, scale):
    c, dt = case, case["proj"].dtype
    rows = c["proj"].shape[0]
    q = torch.empty(rows, c["heads"], c["dk"], device="cuda", dtype=dt)
    att = H().Attention({"heads": c["heads"], "kv_heads": c["kv"], "dk": c["dk"], "dv": c["dv"], "q_off": c["off"][0], "k_off": c["off"][1],
                         "v_off": c["off"][2], "norm_dim": c["dk"], "eps": 1e-5, "scale": scale}, {"q_gamma": gamma_q, "k_gamma": gamma_k})
    att.prep(c["proj"], c["batch"], c["table"], q, c["kc"], c["vc"])
    o = torch.full((rows, c["heads"] * c["dv"]), float("nan"), device="cuda", dtype=dt)
    args = (q, c["kc"], c["vc"], c["batch"], c["table"], c["gate"], o)
    if kernel == "any":
        att.any(*args)
    elif kernel == "prefill":
        att.prefill(*args, max(c["lens"]), status())
    else:
        counters = torch.zeros(4096, dtype=torch.int32, device="cuda")
        for splits in (1, 3):
            scratch = torch.empty(att.decode_scratch(rows, splits), device="cuda")
            att.decode(*args, scratch, counters, splits, status())
            assert int(counters.abs().sum()) == 0
    return q, o.view(rows, c["heads"], c["dv"])


def _attention_want(case, q, scale):
    """From the pages as the append left them (they hold the activation type)."""
    c, out, row = case, [], 0
    d = lambda t: t.double().cpu()
    kc, vc, table = d(c["kc"]), d(c["vc"]), c["table"].cpu()
    for s, n in enumerate(c["lens"]):
        pages = table[s][: (c["total"][s] + 15) // 16].long()
        k, v = kc[pages].flatten(0, 1)[: c["total"][s]], vc[pages].flatten(0, 1)[: c["total"][s]]
        full = torch.zeros(c["total"][s], c["heads"], c["dk"], dtype=torch.float64)
        full[c["bases"][s]:] = d(q[row:row + n])
        o = oracle.causal_attention(full, k, v, scale)[c["bases"][s]:]
        out.append(o * torch.sigmoid(d(c["gate"][row:row + n, : c["heads"]]))[:, :, None])
        row += n
    return torch.cat(out)


@pytest.mark.parametrize("kernel,dtype,heads,kv,dk,dv", [
    ("any", torch.float32, 6, 2, 20, 36), ("any", torch.bfloat16, 3, 3, 40, 130), ("prefill", torch.bfloat16, 4, 2, 64, 128),
    ("prefill", torch.bfloat16, 12, 1, 128, 64), ("prefill", torch.bfloat16, 2, 2, 128, 128), ("decode", torch.bfloat16, 12, 1, 64, 128),
    ("decode", torch.bfloat16, 4, 4, 128, 64), ("decode", torch.bfloat16, 16, 1, 128, 128)])
def test_paged_attention_with_gate(kernel, dtype, heads, kv, dk, dv):
    lens, bases = ([1, 1, 1, 1], [0, 15, 16, 300]) if kernel == "decode" else ([33, 2, 1, 270], [0, 15, 48, 130])
    case = _attention_case(dtype, heads, kv, dk, dv, lens, bases)
    gq, gk = (1 + 0.3 * torch.randn(dk, device="cuda") for _ in range(2))
    scale = 1.3 * dk ** -0.5
    q, o = _run_attention(case, kernel, gq, gk, scale)
    d = lambda t: t.double().cpu()
    p = d(case["proj"])
    rows = p.shape[0]
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2
    close(q, oracle.rms_norm(p[:, : heads * dk].reshape(rows, heads, dk), d(gq), 1e-5), tol)
    # the appended keys and values sit in their pages
    k = oracle.rms_norm(p[:, case["off"][1]: case["off"][1] + kv * dk].reshape(rows, kv, dk), d(gk), 1e-5)
    v = p[:, case["off"][2]: case["off"][2] + kv * dv].reshape(rows, kv, dv)
    seq, pos = case["batch"][3].long().cpu(), case["batch"][4].long().cpu()
    page = case["table"].cpu()[seq, pos // 16].long()
    close(d(case["kc"])[page, pos % 16], k, tol)
    close(d(case["vc"])[page, pos % 16], v, 1e-9)
    close(o, _attention_want(case, q, scale), tol)


@pytest.mark.parametrize("kernel,dk,dv", [("any", 48, 40), ("prefill", 64, 128), ("decode", 64, 128)])
def test_one_key_that_stands_out_is_found_wherever_it_lies(kernel, dk, dv):
    """Key j is the only one that matches its query: the output has to be value j, alone."""
    n, page = 333, 16
    for j in (0, 1, 15, 16, 17, 63, 64, 255, 256, 319, 320, 331, 332):
        lens, bases = ([1], [n - 1]) if kernel == "decode" else ([40], [n - 40])
        case = _attention_case(torch.bfloat16, 2, 1, dk, dv, lens, bases, seed=j)
        case["gate"].fill_(30.0)
        ones = torch.ones(dk, device="cuda")
        at = int(case["table"][0, j // page])
        if j < bases[0]:
            q_row = case["proj"][-1, :dk].float()
            case["kc"][at, j % page, 0] = (q_row / q_row.pow(2).mean().sqrt()).to(torch.bfloat16)
        else:                                              # the last queries ask for a key of the same portion
            case["proj"][j - bases[0], case["off"][1]: case["off"][1] + dk] = case["proj"][-1, :dk]
        _, o = _run_attention(case, kernel, ones, ones, 4.0)
        want = case["vc"][at, j % page, 0].float()
        assert float((o[-1, 0].float() - want).abs().max()) < 0.05, j


def _recurrent_case(kind, heads, kv, dim, vdim, taps, seed, rows, slots=5, dtype=torch.float32, harsh=False):
    g = torch.Generator().manual_seed(seed)
    cq, cv = kv * dim, heads * vdim
    pad = lambda n: (n + 7) // 8 * 8
    off = {"q_off": 0, "k_off": pad(cq), "v_off": 2 * pad(cq), "b_off": 2 * pad(cq) + pad(cv)}
    ld = off["b_off"] + pad(heads)
    spec = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "taps": taps, "delta": int(kind == "delta"),
            "unit_norm": int(kind == "delta"), "decay_kind": int(kind == "delta"), "gate_kind": int(kind == "delta"),
            "q_scale": dim ** -0.5, "inv_tau": 1.0 / 8.0, "eps": 1e-5, **off}
    t = {"state": torch.full((slots, heads, vdim, dim), 7.0), "z_bias": torch.randn(heads * dim, generator=g),
         "gamma": 1 + 0.2 * torch.randn(vdim, generator=g)}
    if kind == "delta":
        t["a_log"] = torch.linspace(-4, 3.0 if harsh else -1.0, heads)
    if taps:
        t["conv_w"] = torch.randn(2 * cq + cv, taps, generator=g) * 0.6
        if taps > 1:
            t["conv_state"] = torch.full((slots, taps - 1, 2 * cq + cv), 7.0)
    t = {k: v.cuda().contiguous() for k, v in t.items()}
    proj = torch.randn(rows, ld, generator=g).to(dtype)
    z = torch.randn(rows, heads * dim, generator=g) * 2
    gate = torch.randn(rows, pad(cv), generator=g).to(dtype)
    return dict(spec=spec, t=t, rec=H().Recurrent(spec, t), proj=proj.cuda(), z=z.cuda(), gate=gate.cuda(), kind=kind)


def _recurrent_want(case, lo, hi):
    """Outputs of rows [lo, hi) run as one sequence from the start, before and after norm and gate."""
    s, t = case["spec"], {k: v.double().cpu() for k, v in case["t"].items()}
    p, z = case["proj"][lo:hi].double().cpu(), case["z"][lo:hi].double().cpu()
    n, Hh, G, dk, dv, taps = hi - lo, s["heads"], s["kv_heads"], s["dim"], s["vdim"], s["taps"]
    q, k = p[:, : G * dk], p[:, s["k_off"]: s["k_off"] + G * dk]
    v = p[:, s["v_off"]: s["v_off"] + Hh * dv]
    if taps:
        w = t["conv_w"]
        q = oracle.silu(oracle.short_conv(q, w[: G * dk]))
        k = oracle.silu(oracle.short_conv(k, w[G * dk: 2 * G * dk]))
        v = oracle.silu(oracle.short_conv(v, w[2 * G * dk:]))
    q, k, v = q.reshape(n, G, dk), k.reshape(n, G, dk), v.reshape(n, Hh, dv)
    z = (z + t["z_bias"]).view(n, Hh, dk)
    if case["kind"] == "delta":
        q, k = oracle.unit(q), oracle.unit(k)
        q, k = (x.repeat_interleave(Hh // G, 1) for x in (q * dk ** -0.5, k))
        beta = torch.sigmoid(p[:, s["b_off"]: s["b_off"] + Hh])
        o = oracle.delta_recurrence(q, k, v, torch.exp(-torch.exp(t["a_log"])[None, :, None] * oracle.softplus(z)), beta)
        act = torch.sigmoid
    else:
        o = oracle.gla_recurrence(q * dk ** -0.5, k, v, torch.sigmoid(z).pow(1.0 / 8.0))
        act = oracle.silu
    g = case["gate"][lo:hi, : Hh * dv].double().cpu().view(n, Hh, dv)
    return o, oracle.rms_norm(o, t["gamma"], 1e-5) * act(g)


def _scan(case, how, rows, lens, bases, slots):
    s, rec = case["spec"], case["rec"]
    batch = ragged(lens, bases, slots)
    n = sum(lens)
    proj, z, gate = case["proj"][rows].contiguous(), case["z"][rows].contiguous(), case["gate"][rows].contiguous()
    out = torch.full((n, (s["heads"] * s["vdim"] + 7) // 8 * 8), float("nan"), device="cuda", dtype=proj.dtype)
    if how == "decode":
        rec.decode(proj, z, gate, 0, 0, batch, out)
        return None, out[:, : s["heads"] * s["vdim"]].view(n, s["heads"], s["vdim"])
    o = torch.full((n, s["heads"], s["vdim"]), float("nan"), device="cuda")
    if how == "seq":
        rec.scan_seq(proj, z, batch, torch.empty(n * (2 * s["kv_heads"] * s["dim"] + s["heads"] * (s["vdim"] + s["dim"] + 1)),
                                                 device="cuda"), o)
    else:
        rec.scan_chunked(proj, z, batch, torch.empty(rec.chunked_scratch(n, len(lens)), device="cuda", dtype=torch.uint8), o,
                         status())
    rec.norm_gate(o, gate, out)
    return o, out[:, : s["heads"] * s["vdim"]].view(n, s["heads"], s["vdim"])


RECURRENT = [("delta", 3, 3, 64, 80, 4, False), ("delta", 6, 2, 44, 28, 3, True), ("delta", 3, 1, 128, 96, 2, True),
             ("delta", 1, 1, 32, 130, 1, False), ("gla", 3, 3, 24, 40, 0, False), ("gla", 2, 2, 128, 128, 0, False),
             ("gla", 2, 2, 64, 17, 0, False), ("delta", 2, 2, 16, 16, 6, True)]


@pytest.mark.parametrize("how,dtype", [("seq", torch.float32), ("seq", torch.bfloat16), ("chunked", torch.bfloat16)])
@pytest.mark.parametrize("kind,heads,kv,dim,vdim,taps,harsh", RECURRENT)
def test_recurrence_portions_and_decoding(how, dtype, kind, heads, kv, dim, vdim, taps, harsh):
    """Three sequences in portions (down to one and two tokens) in slots that hold other values, then decoded
    tokens in a batch of their own. The projections are given, so bf16 engines must reach 32-bit accuracy."""
    rows = 110
    case = _recurrent_case(kind, heads, kv, dim, vdim, taps, seed=dim, rows=rows, dtype=dtype, harsh=harsh)
    spans = [(0, 47), (47, 51), (51, 110)]                  # rows of the three sequences
    want = [_recurrent_want(case, lo, hi) for lo, hi in spans]
    done, slots = [0, 0, 0], [4, 0, 2]
    schedule = [(17, 1, 2), (1, 0, 31), (2, 2, 16), (16, 0, 3), (3, 0, 1)]
    got, raw = [[], [], []], [[], [], []]

    def run(parts, mode):
        live = [i for i in range(3) if parts[i]]
        idx = torch.cat([torch.arange(spans[i][0] + done[i], spans[i][0] + done[i] + parts[i]) for i in live]).cuda()
        o, y = _scan(case, mode, idx, [parts[i] for i in live], [done[i] for i in live], [slots[i] for i in live])
        at = 0
        for i in live:
            got[i].append(y[at:at + parts[i]])
            if o is not None:
                raw[i].append(o[at:at + parts[i]])
            at += parts[i]
            done[i] += parts[i]

    for parts in schedule:
        run(parts, how)
    in_portions = list(done)
    while any(done[i] < spans[i][1] - spans[i][0] for i in range(3)):
        run([int(done[i] < spans[i][1] - spans[i][0]) for i in range(3)], "decode")
    for i in range(3):
        if in_portions[i]:
            close(torch.cat(raw[i]), want[i][0][: in_portions[i]], 3e-5)
        close(torch.cat(got[i]), want[i][1], 3e-5 if dtype == torch.float32 else 1e-2)
    assert all(float((case["t"]["state"][s] - 7.0).abs().max()) == 0 for s in (1, 3))   # other slots untouched


def test_low_rank_maps_inside_the_decode_kernel():
    case = _recurrent_case("delta", 2, 1, 40, 24, 3, seed=3, rows=3, dtype=torch.bfloat16)
    g = torch.Generator().manual_seed(1)
    r = 24
    a2, g2 = (torch.randn(n, r, generator=g).to("cuda", torch.bfloat16) for n in (80, 48))
    spec, t = case["spec"], dict(case["t"], a2=a2, g2=g2)
    rec = H().Recurrent(spec, t)
    ld = case["proj"].shape[1]
    proj = torch.cat([case["proj"], torch.randn(3, 2 * r, generator=g).to("cuda", torch.bfloat16)], 1)
    case["z"] = (proj[:, ld:ld + r].double() @ a2.double().t()).float()
    case["gate"] = (proj[:, ld + r:].double() @ g2.double().t()).float()
    out = torch.empty(3, 48, device="cuda", dtype=torch.bfloat16)
    rec.decode(proj, None, None, ld, ld + r, ragged([1, 1, 1]), out)
    for i in range(3):
        close(out[i].view(2, 24), _recurrent_want(case, i, i + 1)[1][0], 1e-2)


def test_sampler_takes_fp32_logits():
    from mythos_b200.infer.sampler import SamplerConfig, sample

    torch.manual_seed(0)
    lg = torch.randn(5, 3001, device="cuda")
    lg[2, 77] = lg[2].max() * (1 + 1e-6) + 1e-6            # below bf16 resolution
    assert torch.equal(sample(lg, SamplerConfig(temperature=0.0)).long(), lg.argmax(-1))
    t = sample(lg * 50, SamplerConfig(temperature=1.0, top_k=1, top_p=1.0))
    assert torch.equal(t.long(), lg.argmax(-1))


# ------------------------------------------------------------------------------- the engine
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(hu.CONFIGS))
def test_whole_prompt_and_layers(name, dtype):
    cfg = hu.CONFIGS[name]
    w, toks = model_weights(cfg, 2, dtype), hu.tokens(cfg, 75)
    truth = Truth(cfg, w, toks)
    eng = engine(cfg, dtype, w=w)
    seen, run = [], eng._run_layers
    eng._run_layers = lambda i, p, c: run(i, p, c, seen)
    s = eng.cache.new_sequence()
    got = eng.step([s], [toks], [list(range(75))])
    assert len(seen) == len(truth.layers) and all(truth.agrees(x, dtype, layer=i) for i, x in enumerate(seen))
    assert truth.agrees(got, dtype)


@pytest.mark.parametrize("name", sorted(hu.CONFIGS))
@pytest.mark.parametrize("tensor_kernels", [True, False])
def test_portions_and_single_tokens_give_the_whole_prompt(name, tensor_kernels):
    cfg = hu.CONFIGS[name]
    toks = hu.tokens(cfg, 150, 7)
    for dtype in ("float32", "bfloat16"):
        w = model_weights(cfg, 4, dtype)
        truth = Truth(cfg, w, toks)
        eng = engine(cfg, dtype, w=w)
        eng.tensor_kernels = tensor_kernels
        for cuts in ([2, 3, 2, 17, 15, 1, 64, 33, 13], [1] * 40 + [110], [149, 1], [16] * 9 + [6]):
            s, at, out = eng.cache.new_sequence(), 0, []
            for n in cuts:
                out.append(eng.step([s], [toks[at:at + n]], [list(range(n))]))
                at += n
            eng.release(s)
            assert truth.agrees(torch.cat(out), dtype), (dtype, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reuse_pages_and_slots(dtype):
    """Requests of unequal length come and go in a pool that holds two or three of them at a time; portions
    run beside decoded tokens and a request is left out of some steps."""
    for name in ("deep", "ragged", "latent_ragged", "latent_wide", "latent_plain", "scan_ragged", "scan_wide", "scan_plain", "side_ragged",
                 "side_wide", "side_plain"):
        cfg = hu.CONFIGS[name]
        w = model_weights(cfg, 9, dtype)
        eng = engine(cfg, dtype, w=w, kv_pages=22)
        g = torch.Generator().manual_seed(3)
        waiting = [(hu.tokens(cfg, n, n), []) for n in (70, 5, 131, 33, 90, 2, 64, 17)]
        live, finished = [], []
        while waiting or live:
            while waiting and len(live) < 4:
                pages = (len(waiting[0][0]) + 15) // 16
                held = sum((len(r[0]) + 15) // 16 for r in live)
                if held + pages > 22:
                    break
                t, o = waiting.pop(0)
                live.append([t, o, eng.cache.new_sequence(), 0])
            batch = [r for r in live if len(live) == 1 or torch.rand((), generator=g) < 0.75]
            if not batch:
                continue
            parts = []
            for r in batch:
                left = len(r[0]) - r[3]
                n = 1 if r[3] > len(r[0]) // 2 else int(torch.randint(2, 34, (), generator=g))
                parts.append(min(n, left))
            lg = eng.step([r[2] for r in batch], [r[0][r[3]:r[3] + n] for r, n in zip(batch, parts)],
                          [list(range(n)) for n in parts])
            at = 0
            for r, n in zip(batch, parts):
                r[1].append(lg[at:at + n])
                at += n
                r[3] += n
                if r[3] == len(r[0]):
                    eng.release(r[2])
                    finished.append(r)
            live = [r for r in live if r[3] < len(r[0])]
        assert eng.cache.alloc.used == 0 and len(finished) == 8
        for t, o, *_ in finished:
            assert Truth(cfg, w, t).agrees(torch.cat(o), dtype), (name, len(t))


@pytest.mark.parametrize("name", ["wide", "latent_wide", "scan_wide", "side_wide"])
def test_long_decoding_does_not_drift(name):
    cfg = hu.CONFIGS[name]
    toks = hu.tokens(cfg, 420, 5)
    for dtype in ("float32", "bfloat16"):
        w = model_weights(cfg, 6, dtype)
        truth = Truth(cfg, w, toks)
        eng = engine(cfg, dtype, w=w)
        s, twin = eng.cache.new_sequence(), eng.cache.new_sequence()
        out = [eng.step([s, twin], [toks[:20], toks[:35]], [[19], []])]
        for t in toks[20:]:
            out.append(eng.decode([s], [t]))
        assert truth.agrees(torch.cat(out), dtype, slice(19, None))
        lg = eng.step([twin], [toks[35:]])                 # the sequence that waited meanwhile
        assert truth.agrees(lg, dtype, slice(-1, None))


@pytest.mark.parametrize("name", ["deep", "latent_ragged", "scan_ragged", "side_ragged"])
def test_offloaded_sequence_continues_in_another_slot(name):
    cfg = hu.CONFIGS[name]
    w, toks = hu.weights(cfg, 8), hu.tokens(cfg, 60)
    eng = engine(cfg, "float32", w=w)
    a = eng.cache.new_sequence()
    eng.step([a], [toks[:37]])
    handle = eng.cache.offload_sequence(a)
    b = eng.cache.new_sequence()
    eng.step([b], [toks[10:40]])                           # takes the freed slot and pages
    a = eng.cache.restore_sequence(handle)
    got = eng.step([a], [toks[37:]], [list(range(23))])
    assert hu.rel(got, oracle.forward(cfg, w, toks)[37:]) < TOL["float32"]


def _greedy(cfg, w, prompt, n):
    """Greedy continuation by the oracle, and the gap between its two best logits at every step."""
    seq, gaps = list(prompt), []
    for _ in range(n):
        top = torch.topk(oracle.forward(cfg, w, seq)[-1], 2)
        gaps.append(float(top.values[0] - top.values[1]))
        seq.append(int(top.indices[0]))
    return seq[len(prompt):], gaps


@pytest.mark.parametrize("name,wide", [("ragged", "wide"), ("latent_ragged", "latent_wide"), ("scan_ragged", "scan_wide"), ("side_ragged", "side_wide")])
def test_greedy_generation_and_scheduler(name, wide):
    from mythos_b200.infer.sampler import SamplerConfig
    from mythos_b200.infer.serving import ContinuousBatcher

    cfg = hu.CONFIGS[name]
    w = hu.weights(cfg, 1)
    prompts = [hu.tokens(cfg, n, 20 + n) for n in (9, 1, 30)]
    want = []
    for p in prompts:
        out, gaps = _greedy(cfg, w, p, 12)
        assert min(gaps) > 1e-3
        want.append(out)
    eng = engine(cfg, "float32", w=w)
    for graph in (True, False):
        assert eng.generate(prompts, max_new_tokens=12, use_graph=graph).tokens == want
    held = eng.cache.new_sequence()                        # a slot in front is taken
    assert eng.generate(prompts[:2], max_new_tokens=12).tokens == want[:2]
    eng.release(held)
    for chunk in (None, 7):
        cb = ContinuousBatcher(eng, max_batch=2, chunk_tokens=chunk)
        reqs = [cb.submit(p, max_new_tokens=12, sampler=SamplerConfig(temperature=0.0)) for p in prompts]
        cb.run_until_idle()
        assert [r.output for r in reqs] == want
        assert eng.cache.alloc.used == 0
    # bf16: the captured decode graph follows the same path as single steps
    e16 = engine(hu.CONFIGS[wide], seed=3, max_seq_len=640)
    ps = [hu.tokens(hu.CONFIGS[wide], n, n) for n in (40, 40)]
    assert e16.generate(ps, max_new_tokens=20).tokens == e16.generate(ps, max_new_tokens=20, use_graph=False).tokens


@pytest.mark.parametrize("name", ["ragged", "latent_ragged", "scan_ragged", "side_ragged"])
def test_model_helpers_and_command_line(tmp_path, name):
    from mythos_b200.infer.engine import InferenceEngine
    from mythos_b200.infer.serving import compute_logprobs
    from mythos_b200.oil.importers import write_safetensors
    from mythos_b200.oil.model_io import load_model
    from mythos_b200.tools.infer import main as infer_main

    cfg = json.loads(json.dumps(hu.CONFIGS[name]))
    w, toks = model_weights(cfg, 11, "bfloat16"), hu.tokens(cfg, 25)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    m, _ = load_model(str(tmp_path), device="cuda")
    truth = Truth(cfg, w, toks)
    want = truth.logits
    assert truth.agrees(m(torch.tensor([toks]))[0], "bfloat16")
    lp = torch.log_softmax(want, -1)[:-1].gather(1, torch.tensor(toks[1:])[:, None])[:, 0]
    assert float((compute_logprobs(m, toks) - lp).abs().max()) < 0.5
    eng = InferenceEngine.load(str(tmp_path), device="cuda", max_batch=1)
    assert isinstance(eng.generate_text("ab", max_new_tokens=4), str)
    assert infer_main([str(tmp_path), "abc", "-t", "5", "--temperature", "0", "--precision", "fp32"]) == 0
    # the same weights through the trace replay, in another process
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[:4], "want": []}, {"id": "x", "tokens": toks[9:10], "want": [0]}],
              "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[10:], "want": [14]}], "end": ["x"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       text=True, capture_output=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    got = torch.cat([torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32) for i in range(3)])
    assert hu.rel(got.view(4, -1), want[[0, 8, 9, 24]]) < TOL["float32"]


def test_limits_are_errors_not_faults():
    cfg = hu.CONFIGS["single"]
    eng = engine(cfg, max_batch=1, kv_pages=2)
    s = eng.cache.new_sequence()
    with pytest.raises(MemoryError):
        eng.step([s], [hu.tokens(cfg, 33)])
    with pytest.raises(MemoryError):
        eng.cache.new_sequence()
    eng.release(s)
    s = eng.cache.new_sequence()
    with pytest.raises(ValueError):
        eng.step([s], [hu.tokens(cfg, 641)])
    with pytest.raises(ValueError):
        eng.step([s, s], [[1], [2]])

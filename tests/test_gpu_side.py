"""Parallel sublayers on the GPU: input convolution, normalised embedding, residual kernel, PolyNorm, attention whose values
are its keys, window attention over latents with low-rank queries. Each mechanism alone against the plain implementation
in ``hybrid_oracle``; the whole models are covered in ``test_gpu_hybrid``."""
import math

import pytest
import torch

import hybrid_oracle as oracle
import hybrid_util as hu
from test_gpu_hybrid import TOL, H, Truth, close, engine, ragged, status
from test_gpu_latent import Case as Latent
from test_gpu_scan import PAGE, d, pad8, padded

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16


# ------------------------------------------------------------------------------- norms and the stream
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [1, 7, 52, 64, 512, 2048, 2100, 5632, 8192, 8448, 16384, 20000, 32768, 33000])
def test_poly_norm(dtype, width):
    """Rows from tiny to large, so that eps and every power count; into a column range of a wider row."""
    g = torch.Generator().manual_seed(width)
    p, rows = pad8(width), 6
    scale = torch.tensor([1e-3, 0.05, 1.0, 3.0, 20.0, 0.3])[:, None]
    y = (torch.randn(rows, width, generator=g) * scale).to("cuda", dtype)
    bias = (torch.randn(width, generator=g) * 0.3).cuda()
    act = torch.tensor([0.7, -0.5, 0.4, 0.3], device="cuda")
    for b in (bias, None):
        buf = torch.full((rows, 8 + p), 9.0, device="cuda", dtype=dtype)
        H().poly_norm(y, b, act, width, buf[:, 8:], 1e-3)
        want = oracle.poly_norm(d(y) + (d(bias) if b is not None else 0.0), d(act), 1e-3)
        for r in range(rows):
            close(buf[r, 8:8 + width], want[r], 2e-6 if dtype == F32 else 4e-3)
        assert float((buf[:, :8] - 9.0).abs().max()) == 0.0 and float(buf[:, 8 + width:].float().abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,dim,taps", [(3, 100, 3), (1, 64, 1), (5, 333, 2), (4, 2048, 4), (2, 136, 6)])
def test_residual_and_embedding_with_the_next_convolution(dtype, rows, dim, taps):
    """One token of every sequence: stream, norm and convolution in one launch; the convolution starts from zero for a
    sequence without earlier tokens, whatever its slot holds."""
    g = torch.Generator().manual_seed(dim)
    rnd = lambda *s: torch.randn(*s, generator=g).cuda()
    p, tol = pad8(dim), 2e-6 if dtype == F32 else 1e-2
    w, state = rnd(taps, dim) * 0.5, rnd(rows + 2, taps - 1, dim) if taps > 1 else None
    slots, bases = list(range(rows + 2))[::-1][:rows], [0 if i == 1 else 9 for i in range(rows)]
    batch = ragged([1] * rows, bases, slots)
    conv = H().Conv(dim, True, w, state=state)

    def check(call, stream, gamma):
        before = state.clone() if taps > 1 else None
        full = lambda: torch.full((rows, p), float("nan"), device="cuda", dtype=dtype)
        h, out = full(), full()
        x = call(h, (conv, batch, out))
        close(x, stream, 2e-6)
        close(h[:, :dim], oracle.one_number_norm(stream, gamma, 1e-3), tol)
        for i in range(rows):
            past = torch.zeros(taps - 1, dim, dtype=torch.float64) if bases[i] == 0 or taps == 1 else d(before[slots[i]])
            seq = torch.cat([past, d(h[i:i + 1, :dim])])
            close(out[i, :dim], oracle.input_conv(seq, d(w).t())[-1], tol)
            if taps > 1:
                close(state[slots[i]], seq[1:], 1e-7)
        if taps > 1:
            rest = [s for s in range(rows + 2) if s not in slots]
            assert torch.equal(state[rest], before[rest])
        assert float(h[:, dim:].float().abs().sum()) + float(out[:, dim:].float().abs().sum()) == 0.0

    gamma = torch.full((dim,), 1.3, device="cuda")
    for bias in (rnd(dim), None):
        y, x = torch.cat([rnd(rows, dim), rnd(rows, 8)], 1).to(dtype), rnd(rows, dim)
        stream = d(x) + 0.6 * (d(y)[:, :dim] + (d(bias) if bias is not None else 0.0))

        def residual(h, tail):
            H().residual_norm(y, bias, 0.6, x, gamma, h, 1e-3, tail)
            return x

        check(residual, stream, d(gamma))
    emb, ids = rnd(11, dim).to(dtype), torch.randint(0, 11, (rows,), generator=g).to("cuda", torch.int32)
    first = torch.full((dim,), 0.8, device="cuda")

    def embed(h, tail):
        x = torch.empty(rows, dim, device="cuda")
        H().embed_pos_norm(ids, batch[4], emb, None, 1.0, gamma, x, h, 1e-3, first, tail)
        return x

    check(embed, oracle.one_number_norm(d(emb)[ids.long().cpu()], d(first), 1e-3), d(gamma))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim,taps", [(100, 3), (64, 1), (256, 4), (36, 2), (136, 6), (9, 9)])
def test_input_convolution_over_portions(dtype, dim, taps):
    """Three sequences in portions down to one and two tokens, side by side, in slots that hold other values."""
    g = torch.Generator().manual_seed(dim)
    w = torch.randn(dim, taps, generator=g) * 0.5
    state = torch.full((5, taps - 1, dim), 7.0, device="cuda") if taps > 1 else None
    conv = H().Conv(dim, True, w.t().contiguous().cuda(), state=state)
    p = pad8(dim)
    x = padded(torch.randn(3, 90, dim, generator=g), p).to("cuda", dtype)
    slots, done, got = [4, 0, 2], [0, 0, 0], [[], [], []]
    for parts in ((17, 1, 2), (1, 0, 31), (2, 2, 16), (16, 20, 3), (3, 0, 1), (0, 2, 37), (51, 65, 0)):
        live = [i for i in range(3) if parts[i]]
        rows = torch.cat([x[i, done[i]:done[i] + parts[i]] for i in live])
        y = torch.full((rows.shape[0], p), float("nan"), device="cuda", dtype=dtype)
        one = all(parts[i] == 1 for i in live)
        conv.run(rows, 0, ragged([parts[i] for i in live], [done[i] for i in live], [slots[i] for i in live]), one, y)
        assert float(y[:, dim:].float().abs().sum()) == 0.0
        at = 0
        for i in live:
            got[i].append(y[at:at + parts[i], :dim])
            at += parts[i]
            done[i] += parts[i]
    assert done == [90, 90, 90]
    for i in range(3):
        close(torch.cat(got[i]), oracle.input_conv(d(x[i, :, :dim]), d(w)), 2e-6 if dtype == F32 else 8e-3)
    if taps > 1:
        assert all(float((state[s] - 7.0).abs().max()) == 0 for s in (1, 3))


# ------------------------------------------------------------------------------- keys as values
class KeyValues:
    """New tokens of several sequences whose earlier keys and values already lie in shuffled pages."""

    def __init__(self, dtype, heads, kv, dim, rot, lens, bases, seed=0, scale=None, amp=1.0):
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        c = lambda t: t.to("cuda", dtype)
        self.dtype, self.heads, self.kv, self.dim, self.rot, self.lens, self.bases = dtype, heads, kv, dim, rot, lens, bases
        self.scale, self.p, self.amp = 1.3 * dim ** -0.5 if scale is None else scale, pad8(dim), amp
        self.total = [b + n for b, n in zip(bases, lens)]
        need = [(t + PAGE - 1) // PAGE for t in self.total]
        order = torch.randperm(sum(need) + 3, generator=g).tolist()
        table = torch.full((len(lens), max(need) + 1), -1, dtype=torch.int32)
        for s, n in enumerate(need):
            for i in range(n):
                table[s, i] = order.pop()
        self.table, pages, T = table.cuda(), sum(need) + 3, sum(lens)
        self.kc, self.vc = (c(padded(rnd(pages, PAGE, kv, dim), self.p)) for _ in range(2))
        self.proj = c(torch.cat([padded(rnd(T, n, dim), self.p).flatten(1) for n in (heads, kv)], 1))
        self.bq, self.bk = rnd(heads, dim), rnd(kv, dim)
        bq, bk = (padded(b, self.p).flatten().cuda() for b in (self.bq, self.bk))
        turns = torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) / (2 * math.pi) for i in range(rot["dims"] // 2)], dtype=torch.float64)
        off = heads * self.p
        self.att = H().Attention({"heads": heads, "kv_heads": kv, "dk": self.p, "dv": self.p, "scale": self.scale, "k_off": off, "v_off": off,
                                  "rot": rot["dims"], "pairs": 1, "rot_amp": amp, "eps": 1e-2},
                                 {"q_bias": bq, "k_bias": bk, "v_bias": bk, "turns": turns.cuda(), "sink": torch.zeros(heads, device="cuda")})
        self.batch = ragged(lens, bases)
        self.q = torch.full((T, heads, self.p), float("nan"), device="cuda", dtype=dtype)
        self.att.prep(self.proj, self.batch, self.table, self.q, self.kc, self.vc)

    def run(self, how, splits=2):
        T = self.proj.shape[0]
        o = torch.full((T, self.heads * self.p), float("nan"), device="cuda", dtype=self.dtype)
        args = (self.q, self.kc, self.vc, self.batch, self.table, None, o)
        if how == "any":
            self.att.any(*args)
        elif how == "prefill":
            self.att.prefill(*args, max(self.lens), status())
        else:
            counters = torch.zeros(4096, dtype=torch.int32, device="cuda")
            self.att.decode(*args, torch.full((self.att.decode_scratch(T, splits),), float("nan"), device="cuda"), counters, splits, status())
        return o.view(T, self.heads, self.p)[..., : self.dim]

    def rows(self, cache, s):
        n = self.total[s]
        return d(cache)[self.table[s].cpu()[: (n + PAGE - 1) // PAGE].long()].flatten(0, 1)[:n, :, : self.dim]

    def want(self):
        out, at = [], 0
        for s, n in enumerate(self.lens):
            full = torch.zeros(self.total[s], self.heads, self.dim, dtype=torch.float64)
            full[self.bases[s]:] = d(self.q)[at:at + n, :, : self.dim]
            out.append(oracle.banded_attention(full, self.rows(self.kc, s), self.rows(self.vc, s), self.scale, plus_one=True)[self.bases[s]:])
            at += n
        return torch.cat(out)


SHAPES = [(6, 2, 20, 10, 500.0), (4, 4, 64, 64, 1e4), (3, 1, 128, 128, 1e6), (5, 5, 72, 26, 1e4), (2, 1, 136, 72, 300.0), (1, 1, 2, 2, 10.0), (24, 2, 48, 16, 1e5)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SHAPES)
def test_pairs_turn_and_values_are_the_keys_before(dtype, shape):
    """Also far out, where a rounded angle would be off."""
    heads, kv, dim, dims, base = shape
    rot = {"base": base, "dims": dims}
    for amp in (1.0, 1.25):
        c = KeyValues(dtype, heads, kv, dim, rot, lens=[70, 1, 18], bases=[0, 15, 200003], amp=amp)
        T, tol, pos = 89, 3e-6 if dtype == F32 else 9e-3, c.batch[4].cpu()
        raw = d(c.proj)
        q = raw[:, : heads * c.p].view(T, heads, c.p)[..., :dim] + d(c.bq)
        k = raw[:, heads * c.p:].view(T, kv, c.p)[..., :dim] + d(c.bk)
        turned = [oracle.turn_pairs(x, pos, rot) for x in (q, k)]
        for x in turned:
            x[..., :dims] *= amp
        seq = c.batch[3].long().cpu()
        at = c.table.cpu()[seq, pos // PAGE].long(), (pos % PAGE).long()
        close(d(c.q)[..., :dim], turned[0], tol)
        close(d(c.kc)[at][..., :dim], turned[1], tol)
        close(d(c.vc)[at][..., :dim], k, tol)
        assert all(float(x[..., dim:].float().abs().sum()) == 0.0 for x in (c.q, c.kc, c.vc))


@pytest.mark.parametrize("how,dtype,shape", [(h, t, s) for h, t in (("any", F32), ("any", BF16), ("decode", BF16), ("prefill", BF16))
                                             for s in SHAPES if h == "any" or s[2] <= 128])
def test_one_is_added_to_the_denominator(how, dtype, shape):
    heads, kv, dim, dims, base = shape
    lens, bases = ([1] * 5, [0, 15, 16, 300, 63]) if how == "decode" else ([33, 2, 1, 270], [0, 15, 148, 130])
    c = KeyValues(dtype, heads, kv, dim, {"base": base, "dims": dims}, lens, bases)
    want = c.want()
    for splits in ((1, 2, 5) if how == "decode" else (1,)):
        close(c.run(how, splits), want, 2e-5 if dtype == F32 else 2e-2)
    # far below zero the one takes nearly everything, far above nothing
    for shift, share in ((-9.0, 0.0), (9.0, 1.0)):
        c.q.zero_()
        c.q[..., 0], c.kc[..., 0] = shift / c.scale / 4, 4.0
        got = d(c.run(how, 2))
        close(got, c.want(), 2e-2 if dtype == BF16 else 2e-5)
        if share == 0.0 and how == "decode":
            assert float(got[0].abs().max()) < 1e-3 * float(c.rows(c.vc, 0).abs().max()) + 1e-6


# ------------------------------------------------------------------------------- latents
LATENTS = [(3, 20, 6, 36, 44), (20, 128, 64, 128, 256), (17, 72, 2, 40, 512), (2, 64, 32, 64, 64)]


@pytest.mark.parametrize("how,dtype", [("any", F32), ("any", BF16), ("decode", BF16), ("prefill", BF16)])
@pytest.mark.parametrize("window", [1, 16, 64, 65, 130, 1000])
@pytest.mark.parametrize("shape", LATENTS)
def test_gated_window_attention_over_latents(how, dtype, window, shape):
    """Without a sink; long portions take only the latents that the window reaches."""
    lens, bases = ([1] * 6, [0, 15, 16, 300, 63, 129]) if how == "decode" else ([33, 2, 1, 270], [0, 15, 148, 130])
    c = Latent(dtype, *shape, lens=lens, bases=bases, scale=2.0 * (shape[1] + shape[2]) ** -0.5, sink="none", window=window, gate=True)
    c.prep()
    want = c.want()
    for splits in ((1, 2, 5) if how == "decode" else (1,)):
        close(c.run(how, splits), want, 2e-5 if dtype == F32 else 2.5e-2)


@pytest.mark.parametrize("how", ["any", "decode", "prefill"])
def test_one_latent_that_stands_out_at_the_edge_of_a_window(how):
    """Key j alone matches the last query: it is found as long as it lies inside the window, and not one token earlier."""
    n, shape = 333, (2, 40, 24, 40, 64)
    for window in (1, 2, 15, 16, 17, 48, 63, 64, 65, 100, 128, 129, 257, 333, 400):
        for j in {n - window, n - window - 1, n - 1, max(0, n - window // 2 - 1)}:
            if not 0 <= j < n:
                continue
            lens, bases = ([1], [n - 1]) if how == "decode" else ([40], [n - 40])
            c = Latent(BF16, *shape, lens=lens, bases=bases, seed=j, scale=1.5, sink="none", window=window)
            c.prep()
            q, qr = c.queries()
            row = c.cache[int(c.table[0, j // PAGE]), j % PAGE, 0]
            row[c.rank_p: c.rank_p + c.rot] = qr[-1, 0] * 2
            v = d(c.uv[0]) @ d(row[: c.rank])
            got = d(c.run(how, 3))[-1, 0]
            if j >= n - window:
                assert float((got - v).abs().max()) < 0.03 * float(v.abs().max()) + 0.02, (window, j)
            else:
                assert float((got - v).abs().max()) > 0.2, (window, j)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("low", [1, 21, 64, 136])
def test_latents_and_queries_are_prepared_apart(dtype, low):
    """First what queries are a map of and the latents, then the rotated query columns of another matrix; cosines and
    sines grow by their factor."""
    c = Latent(dtype, 3, 20, 6, 36, 44, lens=[5, 1, 18], bases=[0, 15, 200003], amp=1.3)
    T, tol = 24, 2e-6 if dtype == F32 else 9e-3
    g = torch.Generator().manual_seed(low)
    x = torch.randn(T, low, generator=g).to("cuda", dtype)
    off = c.off["kr"] + c.rot_p
    proj = torch.cat([c.raw, padded(x, pad8(low))], 1)
    gamma = (1 + 0.3 * torch.randn(low, generator=g)).cuda()
    spec = {"heads": 3, "rank": 44, "rot": 6, "rank_p": c.rank_p, "rot_p": c.rot_p, "qr_off": 16, "c_off": c.off["c"], "kr_off": c.off["kr"],
            "scale": 1.0, "eps": 1e-5, "rot_amp": 1.3, "low_off": off, "low_rank": low}
    turns = torch.tensor([c.base ** (-2.0 * i / 6) / (2 * math.pi) for i in range(3)], dtype=torch.float64, device="cuda")
    lat = H().Latent(spec, c.gamma, turns, None, gamma)
    lat.prep(proj, c.batch, c.table, c.cache, queries=False)
    close(proj[:, off:off + low], oracle.rms_norm(d(x), d(gamma), 1e-5), tol)
    assert torch.equal(proj[:, :off], c.raw) and float(proj[:, off + low:].float().abs().sum()) == 0.0
    pos, seq = c.batch[4].cpu(), c.batch[3].long().cpu()
    row = d(c.cache)[c.table.cpu()[seq, pos // PAGE].long(), (pos % PAGE).long(), 0]
    raw = d(c.raw)
    close(row[:, :44], oracle.rms_norm(raw[:, c.off["c"]: c.off["c"] + 44], d(c.gamma), 1e-5), tol)
    close(row[:, c.rank_p: c.rank_p + 6], 1.3 * oracle.rotate_pairs(raw[:, c.off["kr"]: c.off["kr"] + 6], pos, c.base), tol)
    cache = c.cache.clone()
    qs = torch.randn(T, 16 + 3 * c.rot_p, generator=g).to("cuda", dtype)
    q0 = d(qs)
    lat.prep(qs, c.batch, c.table, c.cache, latents=False)
    assert torch.equal(c.cache, cache) and torch.equal(d(qs)[:, :16], q0[:, :16])
    want = 1.3 * oracle.rotate_pairs(q0[:, 16:].view(T, 3, c.rot_p)[..., :6], pos, c.base)
    close(d(qs)[:, 16:].view(T, 3, c.rot_p)[..., :6], want, tol)
    # a layer that uses another one's latents touches no page
    shared = H().Latent({k: v for k, v in spec.items() if k not in ("c_off", "kr_off")}, None, turns, None, gamma)
    again = torch.cat([c.raw, padded(x, pad8(low))], 1)
    shared.prep(again, c.batch, c.table, c.cache, queries=False)
    assert torch.equal(c.cache, cache) and torch.equal(again, proj)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_head_products_with_an_output_gate(dtype):
    torch.manual_seed(0)
    for rows in (1, 5, 140):
        x, w = torch.randn(rows, 3, 64, device="cuda").to(dtype), torch.randn(3, 40, 64, device="cuda").to(dtype)
        gate = torch.randn(rows, 136, device="cuda").to(dtype)
        buf = torch.full((rows, 128), 9.0, device="cuda", dtype=dtype)
        H().gemm_heads(x, w, buf[:, :120].unflatten(1, (3, 40)), status(), gate[:, 16:])
        want = torch.einsum("tbk,bnk->tbn", d(x), d(w)).flatten(1) * torch.sigmoid(d(gate)[:, 16:])
        close(buf[:, :120], want, 1e-6 if dtype == F32 else 8e-3)
        assert float((buf[:, 120:] - 9.0).abs().max()) == 0.0


# ------------------------------------------------------------------------------- engine
def test_layers_that_share_latents_hold_one_set():
    cfg = hu.CONFIGS["side_wide"]
    eng = engine(cfg, "float32", w=hu.weights(cfg, 3))
    assert len(eng.cache.k) == 4 and [L.att_index for L in eng.layers] == [0, 1, 2, 1, 3]
    assert [tuple(t.shape[1:]) for t in eng.states.tensors] == [(3, 256)] * 5
    assert eng.cache.share_prefix(eng.cache.new_sequence(), list(range(40))) == 0     # the states are not in the pages


@pytest.mark.parametrize("name", hu.ZIGIVIK)
def test_batch_and_portions_do_not_change_32_bit_logits_beyond_rounding(name):
    """One request alone, beside others, and cut into portions of two tokens."""
    cfg = hu.CONFIGS[name]
    w, toks = hu.weights(cfg, 12), hu.tokens(cfg, 120, 5)
    eng = engine(cfg, "float32", w=w)
    s = eng.cache.new_sequence()
    alone = eng.step([s], [toks], [list(range(120))])
    eng.release(s)
    s, o = eng.cache.new_sequence(), eng.cache.new_sequence()
    beside = eng.step([o, s], [hu.tokens(cfg, 90, 6), toks], [[], list(range(120))])
    eng.release(s)
    s, out = eng.cache.new_sequence(), []
    for i in range(0, 120, 2):
        lists = [toks[i:i + 2]] if i % 3 else [toks[i:i + 2], [i % cfg["vocab"]]]
        out.append(eng.step([s] if i % 3 else [s, o], lists, [[0, 1], []][: len(lists)]))
    for got in (beside, torch.cat(out)):
        assert hu.rel(got, alone) < 2e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_short_and_long_portions_and_single_tokens_in_one_batch(dtype):
    """Every step brings a long portion, a short one and single tokens, at places where windows, pages and key tiles end."""
    cfg = hu.CONFIGS["side_wide"]
    w, eng = hu.weights(cfg, 7), None
    lists = [hu.tokens(cfg, n, n) for n in (260, 140, 90, 75)]
    eng = engine(cfg, dtype, w=w)
    seqs, done, out = [eng.cache.new_sequence() for _ in lists], [0] * 4, [[], [], [], []]
    for parts in ((64, 2, 33, 1), (1, 62, 2, 15), (7, 15, 16, 48), (57, 1, 1, 1), (1, 16, 17, 2), (70, 3, 20, 1), (60, 41, 1, 7)):
        lg = eng.step(seqs, [t[a:a + n] for t, a, n in zip(lists, done, parts)], [list(range(n)) for n in parts])
        for i, x in enumerate(lg.split(list(parts))):
            out[i].append(x)
            done[i] += parts[i]
    assert done == [len(t) for t in lists]
    for t, o in zip(lists, out):
        assert Truth(cfg, w, t).agrees(torch.cat(o), dtype)


@pytest.mark.parametrize("name", ["side_ragged", "side_wide"])
def test_tokens_before_every_window_still_count_through_the_stream(name):
    """An early token that differs changes late logits as the oracle says (full attention sees it), also when the late
    tokens are decoded from pages and slots that another request had used."""
    cfg = hu.CONFIGS[name]
    w = hu.weights(cfg, 15)
    eng = engine(cfg, "float32", w=w, kv_pages=20)
    base = hu.tokens(cfg, 150, 4)
    for first in (base[0], (base[0] + 1) % cfg["vocab"]):
        toks = [first] + base[1:]
        s = eng.cache.new_sequence()
        eng.step([s], [hu.tokens(cfg, 200, first)])
        eng.release(s)
        s = eng.cache.new_sequence()
        out = [eng.step([s], [toks[:141]], [[140]])] + [eng.decode([s], [t]) for t in toks[141:]]
        eng.release(s)
        assert hu.rel(torch.cat(out), Truth(cfg, w, toks).logits[140:]) < TOL["float32"]

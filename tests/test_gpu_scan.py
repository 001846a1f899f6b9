"""Attention with its options (biases, norms, rotation, query temperature, windows, sinks, output gates, shared pages),
selective scans, sigmoid routing and the soft cap on the GPU, each mechanism alone against the plain implementation in
``hybrid_oracle``; the whole models are covered in ``test_gpu_hybrid``."""
import math

import pytest
import torch

import hybrid_oracle as oracle
import hybrid_util as hu
from test_gpu_hybrid import H, close, engine, ragged, status

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
PAGE = 16


def pad8(n):
    return (n + 7) // 8 * 8


def d(t):
    return t.double().cpu()


def padded(t, width):
    """Last dimension filled with zeros up to ``width``."""
    out = t.new_zeros(*t.shape[:-1], width)
    out[..., : t.shape[-1]] = t
    return out


# ------------------------------------------------------------------------------- attention
class Case:
    """New tokens of several sequences whose earlier keys and values already lie in shuffled pages; heads are stored padded
    to a multiple of 8. Unused pages hold other finite values."""

    def __init__(self, dtype, heads, kv, dim, vdim, lens, bases, seed=0, scale=None, window=0, sink=None, gate=None, out_scale=1.0,
                 bias=False, norm=None, rot=None, temp=None, own=True):
        g = torch.Generator().manual_seed(seed)
        self.dtype, self.heads, self.kv, self.dim, self.vdim, self.lens, self.bases = dtype, heads, kv, dim, vdim, lens, bases
        self.window, self.gate_kind, self.out_scale, self.norm, self.rot, self.temp = window, gate, out_scale, norm, rot, temp
        self.scale = 1.3 * dim ** -0.5 if scale is None else scale
        self.dk, self.dv, self.own = pad8(dim), pad8(vdim), own
        self.total = [b + n for b, n in zip(bases, lens)]
        need = [(t + PAGE - 1) // PAGE for t in self.total]
        order = torch.randperm(sum(need) + 3, generator=g).tolist()
        table = torch.full((len(lens), max(need) + 1), -1, dtype=torch.int32)
        for s, n in enumerate(need):
            for i in range(n):
                table[s, i] = order.pop()
        c = lambda t: t.to("cuda", dtype)
        rnd = lambda *s: torch.randn(*s, generator=g)
        pages = sum(need) + 3
        self.kc, self.vc = c(padded(rnd(pages, PAGE, kv, dim), self.dk)), c(padded(rnd(pages, PAGE, kv, vdim), self.dv))
        self.table, T = table.cuda(), sum(lens)
        self.proj = c(torch.cat([padded(rnd(T, n, w), p).flatten(1) for n, w, p in
                                 ((heads, dim, self.dk), (kv, dim, self.dk), (kv, vdim, self.dv))], 1))
        self.gate = None
        if gate == "head":
            self.gate = c(padded(rnd(T, heads), pad8(heads)))
        elif gate == "channel":
            self.gate = c(padded(rnd(T, heads, vdim), self.dv).flatten(1))
        spec = {"heads": heads, "kv_heads": kv, "dk": self.dk, "dv": self.dv, "scale": self.scale, "window": window, "out_scale": out_scale,
                "gate_channels": int(gate == "channel"), "norm_dim": dim if norm else 0, "eps": 1e-2}
        if own:
            spec.update(k_off=heads * self.dk, v_off=(heads + kv) * self.dk)
        self.t = {}
        if sink is not None:
            self.t["sink"] = torch.full((heads,), float(sink)) if not isinstance(sink, str) else rnd(heads) * 1.5
        if bias:
            for n, k, w, p in (("q", heads, dim, self.dk), ("k", kv, dim, self.dk), ("v", kv, vdim, self.dv)):
                self.t[n + "_bias"] = padded(rnd(k, w), p).flatten()
        if norm == "weighted":
            self.t["q_gamma"], self.t["k_gamma"] = (padded(1 + 0.3 * rnd(dim), self.dk) for _ in range(2))
        if rot:
            spec["rot"] = rot["dims"]
            self.t["turns"] = torch.tensor([f / (2 * math.pi) for f in oracle.frequencies(rot)], dtype=torch.float64)
        if temp:
            spec.update(temp_coef=temp["coef"], temp_every=temp["every"])
        self.t = {k: v.cuda() for k, v in self.t.items()}
        self.att, self.batch = H().Attention(spec, self.t), ragged(lens, bases)

    def prep(self):
        self.q = torch.full((self.proj.shape[0], self.heads, self.dk), float("nan"), device="cuda", dtype=self.dtype)
        self.att.prep(self.proj, self.batch, self.table, self.q, self.kc, self.vc)
        return self.q

    def rows(self, cache, s):
        n = self.total[s]
        return d(cache)[self.table[s].cpu()[: (n + PAGE - 1) // PAGE].long()].flatten(0, 1)[:n]

    def run(self, how, splits=3, ldo=0):
        T, width = self.proj.shape[0], self.heads * self.dv
        buf = torch.full((T, width + ldo), 7.0, device="cuda", dtype=self.dtype)
        o = buf[:, :width]
        args = (self.q, self.kc, self.vc, self.batch, self.table, self.gate, o)
        if how == "any":
            self.att.any(*args)
        elif how == "prefill":
            self.att.prefill(*args, max(self.lens), status())
        else:
            counters = torch.zeros(4096, dtype=torch.int32, device="cuda")
            self.att.decode(*args, torch.full((self.att.decode_scratch(T, splits),), float("nan"), device="cuda"), counters, splits, status())
            assert int(counters.abs().sum()) == 0
        assert ldo == 0 or float((buf[:, width:] - 7.0).abs().max()) == 0.0
        return o.view(T, self.heads, self.dv) if ldo == 0 else o.reshape(T, self.heads, self.dv)

    def want(self):
        """From queries and pages as they are."""
        out, at = [], 0
        sink = d(self.t["sink"]) if "sink" in self.t else None
        for s, n in enumerate(self.lens):
            full = torch.zeros(self.total[s], self.heads, self.dim, dtype=torch.float64)
            full[self.bases[s]:] = d(self.q)[at:at + n, :, : self.dim]
            k, v = self.rows(self.kc, s)[..., : self.dim], self.rows(self.vc, s)[..., : self.vdim]
            out.append(oracle.window_sink_attention(full, k, v, self.scale, self.window or None, sink)[self.bases[s]:])
            at += n
        o = torch.cat(out) * self.out_scale
        if self.gate_kind == "head":
            o = o * torch.sigmoid(d(self.gate)[:, : self.heads, None])
        elif self.gate_kind == "channel":
            o = o * torch.sigmoid(d(self.gate).view(-1, self.heads, self.dv)[..., : self.vdim])
        return o


PREP = [  # heads, kv, dim, vdim, options
    (6, 2, 20, 36, dict(bias=True, norm="plain", temp={"coef": 0.4, "every": 16})),
    (4, 4, 64, 64, dict(rot={"base": 500.0, "dims": 64, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}})),
    (3, 1, 128, 40, dict(rot={"base": 1e6, "dims": 10}, norm="weighted", bias=True)),
    (5, 5, 72, 128, dict(rot={"base": 1e4, "dims": 48}, temp={"coef": 1.5, "every": 3})),
    (2, 1, 160, 136, dict(rot={"base": 1e4, "dims": 160}, bias=True, norm="plain", temp={"coef": 0.2, "every": 1})),
    (1, 1, 2, 8, dict(rot={"base": 10.0, "dims": 2})),
    (40, 8, 48, 24, dict(norm="weighted")),
]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("case", PREP)
def test_projection_to_queries_and_cached_keys(dtype, case):
    """Bias, norm, rotation and temperature, also far out, where a rounded angle would be off, and at the steps of the
    temperature."""
    heads, kv, dim, vdim, opt = case
    c = Case(dtype, heads, kv, dim, vdim, lens=[70, 1, 18], bases=[0, 15, 200003], **opt)
    q = c.prep()
    T, tol, pos = sum(c.lens), 3e-6 if dtype == F32 else 9e-3, c.batch[4].cpu()
    raw = d(c.proj)
    part = lambda off, n, w, p: raw[:, off:off + n * p].view(T, n, p)[..., :w]
    parts = {"q": part(0, heads, dim, c.dk), "k": part(heads * c.dk, kv, dim, c.dk), "v": part((heads + kv) * c.dk, kv, vdim, c.dv)}
    for n, x in parts.items():
        if n + "_bias" in c.t:
            x = x + d(c.t[n + "_bias"]).view(x.shape[1], -1)[:, : x.shape[2]]
        if n != "v":
            if c.norm:
                x = oracle.rms(x, 1e-2) * (d(c.t[n + "_gamma"])[:dim] if c.norm == "weighted" else 1.0)
            if c.rot:
                x = oracle.rotate_halves(x, pos, c.rot)
        parts[n] = x
    if c.temp:
        parts["q"] = parts["q"] * oracle.query_temperature(pos, c.temp)[:, None, None]
    close(d(q)[..., :dim], parts["q"], tol)
    seq = c.batch[3].long().cpu()
    at = c.table.cpu()[seq, pos // PAGE].long(), (pos % PAGE).long()
    close(d(c.kc)[at][..., :dim], parts["k"], tol)
    close(d(c.vc)[at][..., :vdim], parts["v"], tol)
    pads = (q[..., dim:], c.kc[..., dim:], c.vc[..., vdim:])
    assert all(float(x.float().abs().sum()) == 0.0 for x in pads)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_shared_keys_and_values_are_left_alone(dtype):
    c = Case(dtype, 4, 2, 24, 16, lens=[9, 1], bases=[3, 40], norm="plain", own=False)
    k0, v0 = c.kc.clone(), c.vc.clone()
    q = c.prep()
    assert torch.equal(c.kc, k0) and torch.equal(c.vc, v0)
    close(d(q), oracle.rms(d(c.proj)[:, :96].view(10, 4, 24), 1e-2), 1e-5 if dtype == F32 else 9e-3)


SHAPES = [(6, 2, 20, 36), (1, 1, 64, 64), (12, 1, 72, 104), (4, 4, 96, 24), (16, 2, 128, 128), (9, 3, 8, 72)]
OPTIONS = [dict(window=19, sink="random"), dict(gate="channel", out_scale=0.7), dict(window=1, gate="head"), dict(window=130, sink=2.0, out_scale=-1.5),
           dict(window=64, gate="channel", sink="random")]


@pytest.mark.parametrize("how,dtype", [("any", F32), ("any", BF16), ("decode", BF16), ("prefill", BF16)])
@pytest.mark.parametrize("opt", OPTIONS)
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_options(how, dtype, opt, shape):
    """Windows shorter and longer than a page, a key tile and a query tile; into rows of a wider buffer."""
    lens, bases = ([1] * 6, [0, 15, 16, 300, 63, 129]) if how == "decode" else ([33, 2, 1, 300], [0, 15, 148, 130])
    c = Case(dtype, *shape, lens=lens, bases=bases, **opt)
    c.prep()
    want = c.want()
    for splits in ((1, 2, 5, 32) if how == "decode" else (1,)):
        got = c.run(how, splits, ldo=8)
        close(got[..., : c.vdim], want, 2e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("how", ["any", "decode", "prefill"])
@pytest.mark.parametrize("sink", [-30.0, 0.0, 4.0, 300.0])
def test_sink_takes_its_share(how, sink):
    lens, bases = ([1, 1], [0, 100]) if how == "decode" else ([20, 17], [0, 90])
    c = Case(BF16, 3, 3, 32, 40, lens=lens, bases=bases, sink=sink, window=50)
    c.prep()
    got, want = c.run(how, 2)[..., :40], c.want()
    assert float((d(got) - want).abs().max()) < 0.02 * max(0.05, float(want.abs().max()))
    if sink == 300.0:
        assert float(got.abs().max()) == 0.0


@pytest.mark.parametrize("how", ["any", "decode", "prefill"])
def test_low_scores_behind_masked_tiles(how):
    """Scores far below zero for every key a query sees: rows that see nothing of a tile's first keys must not fix their
    running maximum there."""
    lens, bases = ([1, 1], [250, 700]) if how == "decode" else ([256], [300])
    c = Case(BF16, 1, 1, 64, 64, lens=lens, bases=bases, window=40, scale=1.0)
    c.prep()
    c.q.zero_()
    c.q[..., 0] = 20.0
    c.kc[..., 0] = -20.0 + 0.125 * torch.randn(c.kc.shape[:-1], device="cuda").to(BF16)
    close(c.run(how, 3), c.want(), 2e-2)


@pytest.mark.parametrize("how,dim,vdim", [("any", 48, 40), ("prefill", 64, 128), ("prefill", 72, 24), ("decode", 64, 128), ("decode", 40, 96)])
def test_one_key_that_stands_out_at_the_edge_of_a_window(how, dim, vdim):
    """Key j alone matches the last query: it is found as long as it lies inside the window, and not one token earlier."""
    n = 333
    for window in (1, 2, 15, 16, 17, 31, 48, 63, 64, 65, 100, 128, 129, 256, 257, 333, 400):
        for j in {n - window, n - window - 1, n - 1, max(0, n - window // 2 - 1)}:
            if not 0 <= j < n:
                continue
            lens, bases = ([1], [n - 1]) if how == "decode" else ([140], [n - 140])
            c = Case(BF16, 2, 1, dim, vdim, lens=lens, bases=bases, seed=j, window=window, scale=2.0)
            c.prep()
            at = int(c.table[0, j // PAGE]), j % PAGE, 0
            c.kc[at] = c.q[-1, 0] * 1.5
            got, v = d(c.run(how, 3))[-1, 0, :vdim], d(c.vc[at])[:vdim]
            if j >= n - window:
                assert float((got - v).abs().max()) < 0.05, (window, j)
            else:
                assert float((got - v).abs().max()) > 0.2, (window, j)
                close(got, c.want()[-1, 0], 2e-2)


# ------------------------------------------------------------------------------- selective scan
class Scan:
    def __init__(self, dtype, inner, state, rank, taps, rows, slots=5, seed=0, out_scale=0.8):
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.dtype, self.inner, self.state, self.rank, self.taps, self.out_scale = dtype, inner, state, rank, taps, out_scale
        p, sp = pad8(inner), H().selective_padded_state(state)
        self.z_off, self.b_off = p, pad8(rank)
        self.c_off = self.b_off + pad8(state)
        c = lambda t: t.to("cuda", dtype)
        self.proj = c(torch.cat([padded(rnd(rows, inner), p), padded(rnd(rows, inner), p)], 1))
        self.w_low = c(torch.cat([padded((rnd(n, inner) * 1.5 * inner ** -0.5).t(), pad8(n)).t() for n in (rank, state, state)]))
        self.w_dt = c(padded(rnd(inner, rank) * rank ** -0.5, pad8(rank)))
        self.A = -torch.exp(rnd(inner, state) * 1.5 - 0.5)
        a = torch.zeros(inner, sp)
        a[:, :state] = self.A.double() / math.log(2.0)
        self.conv_w, self.conv_b, self.D, self.dt_b = rnd(inner, taps) * 0.5, rnd(inner) * 0.3, 1 + 0.3 * rnd(inner), rnd(inner) * 1.5 - 2.0
        self.t = {"a": a, "d": self.D, "dt_b": self.dt_b,
                  "state": torch.full((slots, inner, sp), 7.0)}
        self.t = {k: v.contiguous().cuda() for k, v in self.t.items()}
        self.t["w_dt"] = self.w_dt
        self.conv = H().Conv(inner, False, self.conv_w.t().contiguous().cuda(), self.conv_b.cuda(),
                             torch.full((slots, taps - 1, inner), 7.0, device="cuda") if taps > 1 else None)
        self.sel = H().Selective({"inner": inner, "state": state, "rank": rank, "out_scale": out_scale, "z_off": self.z_off,
                                  "b_off": self.b_off, "c_off": self.c_off}, self.t)

    def want(self, lo, hi):
        """Rows [lo, hi) as one sequence from the start; the convolved channels and the maps are rounded as the kernels
        store them."""
        r = lambda t: d(t.to(self.dtype))
        p = d(self.proj[lo:hi])
        x = r(oracle.silu(oracle.short_conv(p[:, : self.inner], d(self.conv_w)) + d(self.conv_b)))
        low = r(x @ d(self.w_low)[:, : self.inner].t())
        dt = oracle.softplus(low[:, : self.rank] @ d(self.w_dt)[:, : self.rank].t() + d(self.dt_b))
        B, C = (low[:, o:o + self.state] for o in (self.b_off, self.c_off))
        y = oracle.selective_scan(x, dt, d(self.A), B, C, d(self.D))
        return y * oracle.silu(p[:, self.z_off:self.z_off + self.inner]) * self.out_scale

    def run(self, idx, lens, bases, slots, one):
        """One step over rows ``idx`` of the projection, one token per sequence in the single-token form."""
        proj, batch, n = self.proj[idx].contiguous(), ragged(lens, bases, slots), sum(lens)
        full = lambda *s, t=self.dtype: torch.full(s, float("nan"), device="cuda", dtype=t)
        x = full(n, pad8(self.inner))
        self.conv.run(proj, 0, batch, one, x)
        assert float(x[:, self.inner:].float().abs().sum()) == 0.0
        low = (d(x)[:, : self.inner] @ d(self.w_low)[:, : self.inner].t()).to("cuda", self.dtype)
        dt = (d(low)[:, : self.rank] @ d(self.w_dt)[:, : self.rank].t()).float().cuda()
        buf = torch.full((n, 8 + pad8(self.inner)), 9.0, device="cuda", dtype=self.dtype)
        out = buf[:, 8:]
        if one:
            self.sel.step(proj, x, low, dt if n > 2 else None, batch, out)
        else:
            scratch = full(self.sel.scratch_floats(len(lens), n, max(lens)), t=F32)
            self.sel.scan(proj, x, low, dt, batch, max(lens), scratch, out, status())
        assert float((buf[:, :8] - 9.0).abs().max()) == 0.0
        return out[:, : self.inner].clone()


SCANS = [(52, 5, 3, 3), (256, 16, 16, 4), (8, 1, 1, 1), (100, 24, 40, 4), (40, 130, 24, 6), (24, 40, 8, 2), (9, 12, 5, 9), (16, 300, 8, 4)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("sizes", SCANS)
def test_selective_scan_portions_and_decoding(dtype, sizes):
    """Three sequences in portions (down to one and two tokens, and long enough to be cut into chunks) in slots that hold
    other values, then decoded tokens in batches of their own."""
    rows = 420
    c = Scan(dtype, *sizes, rows=rows, seed=sizes[0])
    spans = [(0, 47), (47, 51), (51, rows)]
    want = [c.want(lo, hi) for lo, hi in spans]
    done, slots, got = [0, 0, 0], [4, 0, 2], [[], [], []]

    def run(parts, one):
        live = [i for i in range(3) if parts[i]]
        idx = torch.cat([torch.arange(spans[i][0] + done[i], spans[i][0] + done[i] + parts[i]) for i in live]).cuda()
        y = c.run(idx, [parts[i] for i in live], [done[i] for i in live], [slots[i] for i in live], one)
        at = 0
        for i in live:
            got[i].append(y[at:at + parts[i]])
            at += parts[i]
            done[i] += parts[i]

    for parts in ((17, 1, 2), (1, 0, 31), (2, 2, 16), (16, 0, 3), (3, 0, 1), (0, 0, 290), (2, 0, 2)):
        run(parts, False)
    while any(done[i] < spans[i][1] - spans[i][0] for i in range(3)):
        run([int(done[i] < spans[i][1] - spans[i][0]) for i in range(3)], True)
    for i in range(3):
        # bf16: the output itself, and now and then the other neighbour where the stored channels are rounded
        close(torch.cat(got[i]), want[i], 3e-5 if dtype == F32 else 1.5e-2)
    assert all(float((c.t["state"][s] - 7.0).abs().max()) == 0 for s in (1, 3))      # other slots untouched


def test_chunks_and_whole_portions_give_the_same_states():
    """2000 tokens alone (many chunks) and beside 60 others of the same length (one pass each): outputs and final states."""
    c = Scan(F32, 128, 16, 8, 4, rows=2000, slots=66)
    idx = torch.arange(2000).cuda()
    alone = c.run(idx, [2000], [0], [0], False)
    assert c.sel.scratch_floats(1, 2000, 2000) > 0 and c.sel.scratch_floats(130, 130 * 2000, 2000) == 0
    many = c.run(idx.repeat(64), [2000] * 64, [0] * 64, list(range(1, 65)), False)
    for s in (0, 31, 63):
        close(many[s * 2000:(s + 1) * 2000], alone, 2e-5)
        close(c.t["state"][s + 1], c.t["state"][0], 2e-5)
    close(alone, c.want(0, 2000), 3e-5)


def test_a_far_token_is_remembered_and_a_fast_decay_forgets():
    """One token with a large step; channels with A near zero carry it 1500 tokens, those with a large A lose it."""
    n, c = 1500, Scan(F32, 64, 4, 8, 1, rows=1500)
    a = c.t["a"].view(64, -1, 4)
    a[:32], a[32:] = -1e-6, -20.0
    c.A = (a.reshape(64, -1)[:, :4] * math.log(2.0)).cpu()
    c.proj[1:, :64] *= 1e-3
    c.proj[0, :64] = 5.0
    y = c.run(torch.arange(n).cuda(), [n], [0], [1], False)
    want = c.want(0, n)
    close(y, want, 1e-4)
    state = c.t["state"][1, :, :4].abs().amax(1)
    assert float(state[:32].min()) > 1e-2 and float(state[32:].max()) < 1e-2 * float(state[:32].max())


# ------------------------------------------------------------------------------- routing and output
@pytest.mark.parametrize("E,top,groups,keep,scale,T", [(12, 3, 4, 2, 1.7, 50), (1, 1, 1, 1, 2.0, 3), (64, 6, 8, 3, 2.5, 300), (100, 7, 5, 5, 0.3, 33),
                                                       (8, 8, 2, 2, 1.0, 9), (256, 8, 8, 4, 1.0, 1), (40, 1, 40, 1, 1.5, 70), (16, 4, 2, 1, 1.0, 40)])
def test_sigmoid_routing(E, top, groups, keep, scale, T):
    """Groups by their two best scores, normalised weights; groups of one expert count that one."""
    g = torch.Generator().manual_seed(E + T)
    z = torch.randn(T, E, generator=g) * 2
    i32 = dict(device="cuda", dtype=torch.int32)
    idx, slot = (torch.full((T, top), -1, **i32) for _ in range(2))
    weight = torch.full((T, top), float("nan"), device="cuda")
    counts, offset, count = torch.zeros(E + 1, **i32), torch.full((E,), -1, **i32), torch.full((1,), -1, **i32)
    tiles = torch.full((min(T * top, E + T * top // 16), 3), -1, **i32)
    H().expert_select(z.cuda(), None, (E, top, groups, keep), 16, idx, weight, slot, counts, offset, tiles, count, (1, 2, 1, scale))
    r = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}
    for t in range(T):
        want = dict(oracle.choose_by_sigmoid(z[t].double(), r))
        got = dict(zip(idx[t].tolist(), weight[t].tolist()))
        assert sorted(got) == sorted(want)
        assert all(abs(got[e] - float(w)) < 2e-6 * scale + 1e-7 for e, w in want.items())
    places = (offset[idx.long()] + slot).flatten()
    assert sorted(places.tolist()) == list(range(T * top)) and int(counts.abs().sum()) == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim", [100, 333, 2048])
def test_experts_with_a_shared_one(dtype, dim):
    g = torch.Generator().manual_seed(dim)
    T, top, ld = 7, 3, pad8(dim)
    c = lambda t: t.to("cuda", dtype)
    y, shared = c(torch.randn(T * top, ld, generator=g)), c(torch.randn(T, ld, generator=g) * 2)
    row = torch.randperm(T * top, generator=g).view(T, top).to("cuda", torch.int32)
    w = torch.rand(T, top, generator=g).cuda()
    post, nxt = (1 + 0.3 * torch.randn(dim, generator=g).cuda() for _ in range(2))
    x = torch.randn(T, dim, generator=g).cuda()
    x0, h = d(x), torch.full((T, ld), float("nan"), device="cuda", dtype=dtype)
    H().expert_norm(y, shared, row, w, post, x, nxt, h, 1e-4)
    total = (d(y)[row.cpu().long()] * d(w)[..., None]).sum(1)[:, :dim] + d(shared)[:, :dim]
    want = x0 + oracle.rms_norm(total, d(post), 1e-4)
    close(x, want, 1e-5)
    close(h[:, :dim], oracle.rms_norm(want, d(nxt), 1e-4), 1e-5 if dtype == F32 else 6e-3)


def test_soft_cap():
    torch.manual_seed(0)
    y = torch.randn(5, 333, device="cuda") * 30
    y0 = d(y)
    H().soft_cap(y, 12.5)
    close(y, oracle.soft_cap(y0, 12.5), 1e-6)
    for M in (1, 40):
        x, w = torch.randn(M, 128, device="cuda").to(BF16), torch.randn(200, 128, device="cuda").to(BF16)
        out = torch.empty(M, 200, device="cuda")
        H().gemm_decode(x, w, out, 0, 0, 0.5, status(), cap=3.0)
        close(out, oracle.soft_cap(0.5 * d(x) @ d(w).t(), 3.0), 1e-5)


# ------------------------------------------------------------------------------- engine
def test_layers_that_share_pages_hold_one_set():
    cfg = hu.CONFIGS["scan_ragged"]
    eng = engine(cfg, "float32", w=hu.weights(cfg, 3))
    assert len(eng.cache.k) == 2 and [L.att_index for L in eng.layers] == [0, 1, 0]
    assert eng.cache.share_prefix(eng.cache.new_sequence(), list(range(40))) == 0     # the states are not in the pages


@pytest.mark.parametrize("name", ["scan_wide", "scan_plain"])
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
        lists = [toks[i:i + 2]] if i % 3 else [toks[i:i + 2], [i]]
        out.append(eng.step([s] if i % 3 else [s, o], lists, [[0, 1], []][: len(lists)]))
    for other in (beside, torch.cat(out)):
        assert hu.rel(other, alone) < 2e-5

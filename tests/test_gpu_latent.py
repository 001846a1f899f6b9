"""Latent attention, routed experts and the token input on the GPU, each mechanism alone against the plain
implementation in ``hybrid_oracle``; the whole models are covered in ``test_gpu_hybrid``."""
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


# ------------------------------------------------------------------------------- latent attention
class Case:
    """New tokens of several sequences whose earlier tokens already lie in shuffled pages. ``proj`` holds unrotated
    queries | rotated queries | latent | key part as the layer's projection leaves them. ``sink``: a number for every head,
    "none", or None for random ones."""

    def __init__(self, dtype, heads, dim, rot, vdim, rank, lens, bases, seed=0, base=10000.0, scale=None, sink=None, window=0,
                 gate=False, amp=1.0):
        g = torch.Generator().manual_seed(seed)
        self.dtype, self.heads, self.dim, self.rot, self.vdim, self.rank = dtype, heads, dim, rot, vdim, rank
        self.lens, self.bases, self.base, self.window, self.amp = lens, bases, base, window, amp
        self.scale = (dim + rot) ** -0.5 if scale is None else scale
        self.rank_p, self.rot_p, self.dim_p, self.vdim_p = pad8(rank), pad8(rot), pad8(dim), pad8(vdim)
        self.total = [b + n for b, n in zip(bases, lens)]
        need = [(t + PAGE - 1) // PAGE for t in self.total]
        order = torch.randperm(sum(need) + 3, generator=g).tolist()
        table = torch.full((len(lens), max(need) + 1), -1, dtype=torch.int32)
        for s, n in enumerate(need):
            for i in range(n):
                table[s, i] = order.pop()
        self.W = self.rank_p + self.rot_p
        cache = torch.zeros(sum(need) + 3, PAGE, 1, self.W)
        cache[..., :rank] = torch.randn(*cache.shape[:3], rank, generator=g)
        cache[..., self.rank_p: self.rank_p + rot] = torch.randn(*cache.shape[:3], rot, generator=g)
        T = sum(lens)
        self.off = {"q": 0, "qr": heads * self.dim_p, "c": heads * (self.dim_p + self.rot_p)}
        self.off["kr"] = self.off["c"] + self.rank_p
        proj = torch.zeros(T, self.off["kr"] + self.rot_p)
        proj[:, : self.off["qr"]].view(T, heads, self.dim_p)[..., :dim] = torch.randn(T, heads, dim, generator=g)
        proj[:, self.off["qr"]: self.off["c"]].view(T, heads, self.rot_p)[..., :rot] = torch.randn(T, heads, rot, generator=g)
        proj[:, self.off["c"]: self.off["c"] + rank] = torch.randn(T, rank, generator=g)
        proj[:, self.off["kr"]: self.off["kr"] + rot] = torch.randn(T, rot, generator=g)
        c = lambda t: t.to("cuda", dtype)
        self.table, self.cache, self.proj = table.cuda(), c(cache), c(proj)
        self.gamma = (1 + 0.3 * torch.randn(rank, generator=g)).cuda()
        self.sink = None
        if sink != "none":
            self.sink = (torch.randn(heads, generator=g) * 1.5 if sink is None else torch.full((heads,), float(sink))).cuda()
        self.uk = c(torch.randn(heads, dim, rank, generator=g) * rank ** -0.5)
        self.uv = c(torch.randn(heads, vdim, rank, generator=g) * rank ** -0.5)
        turns = torch.tensor([base ** (-2.0 * i / rot) / (2 * math.pi) for i in range(rot // 2)], dtype=torch.float64)
        self.lat = H().Latent({"heads": heads, "rank": rank, "rot": rot, "rank_p": self.rank_p, "rot_p": self.rot_p,
                               "qr_off": self.off["qr"], "c_off": self.off["c"], "kr_off": self.off["kr"], "scale": self.scale,
                               "eps": 1e-5, "window": window, "rot_amp": amp}, self.gamma, turns.cuda(), self.sink)
        self.batch = ragged(lens, bases)
        self.raw = self.proj.clone()
        self.gate = None
        if gate:
            self.gate = torch.zeros(T, 8 + heads * self.vdim_p)
            self.gate[:, 8:].view(T, heads, self.vdim_p)[..., :vdim] = torch.randn(T, heads, vdim, generator=g)
            self.gate = c(self.gate)[:, 8:]

    def prep(self):
        self.lat.prep(self.proj, self.batch, self.table, self.cache)

    def rows(self, s):
        """Cached rows of sequence s in order."""
        return d(self.cache)[self.table[s].cpu()[: (self.total[s] + PAGE - 1) // PAGE].long()].flatten(0, 1)[: self.total[s], 0]

    def queries(self):
        T = self.proj.shape[0]
        q = self.proj[:, : self.off["qr"]].view(T, self.heads, self.dim_p)
        return q, self.proj[:, self.off["qr"]: self.off["c"]].view(T, self.heads, self.rot_p)

    def run(self, how, splits=1):
        T, Hn = self.proj.shape[0], self.heads
        out = torch.full((T, Hn, self.vdim_p), float("nan"), device="cuda", dtype=self.dtype)
        q, _ = self.queries()
        if how == "prefill":
            first = [max(0, b - self.window + 1) if self.window else 0 for b in self.bases]
            held = [t - f for t, f in zip(self.total, first)]
            keys, i32 = sum(held), dict(dtype=torch.int32, device="cuda")
            cu = torch.tensor([sum(held[:i]) for i in range(len(held) + 1)], **i32)
            lat = torch.full((keys, self.W), float("nan"), device="cuda", dtype=self.dtype)
            self.lat.gather(self.table, self.cache, cu, torch.tensor(first, **i32), max(held), lat)
            kv = torch.zeros(keys, Hn * (self.dim_p + self.vdim_p), device="cuda", dtype=self.dtype)
            k, v = kv[:, : Hn * self.dim_p].unflatten(1, (Hn, self.dim_p)), kv[:, Hn * self.dim_p:].unflatten(1, (Hn, self.vdim_p))
            c = lat[:, : self.rank].float()
            k[..., : self.dim] = torch.einsum("tr,hdr->thd", c, self.uk.float()).to(self.dtype)
            v[..., : self.vdim] = torch.einsum("tr,hdr->thd", c, self.uv.float()).to(self.dtype)
            self.lat.attn_prefill(q, self.proj, k, v, lat, self.batch, cu, torch.tensor(held, **i32), max(self.lens), 1, self.gate,
                                  out, status())
            return out[..., : self.vdim]
        uk = torch.zeros(Hn, self.rank_p, self.dim_p, device="cuda", dtype=self.dtype)
        uk[:, : self.rank, : self.dim] = self.uk.transpose(1, 2)
        uv = torch.zeros(Hn, self.vdim_p, self.rank_p, device="cuda", dtype=self.dtype)
        uv[:, : self.vdim, : self.rank] = self.uv
        ql = torch.full((T, Hn, self.rank_p), float("nan"), device="cuda", dtype=self.dtype)
        ol = torch.full_like(ql, float("nan"))
        H().gemm_heads(q, uk, ql, status())
        if how == "any":
            self.lat.attn_any(ql, self.proj, self.batch[3], self.batch[4], self.table, self.cache, ol)
        else:
            assert self.lat.decode_ok(PAGE)
            scratch = torch.full((T * Hn * splits * (self.rank_p + 4),), float("nan"), device="cuda")
            self.lat.attn_decode(ql, self.proj, self.batch[3], self.batch[4], self.table, self.cache, ol, scratch, splits, status())
        H().gemm_heads(ol, uv, out, status(), self.gate)
        return out[..., : self.vdim]

    def want(self):
        """From the cached rows as they are, with the rotated queries of the projection."""
        out, at = [], 0
        q, qr = self.queries()
        q = torch.cat([d(q)[..., : self.dim], d(qr)[..., : self.rot]], -1)
        uk, uv = d(self.uk), d(self.uv)
        for s, n in enumerate(self.lens):
            rows = self.rows(s)
            c, kr = rows[:, : self.rank], rows[:, self.rank_p: self.rank_p + self.rot]
            k = torch.cat([torch.einsum("tr,hdr->thd", c, uk), kr[:, None].expand(-1, self.heads, -1)], -1)
            v = torch.einsum("tr,hdr->thd", c, uv)
            full = torch.zeros(self.total[s], self.heads, q.shape[-1], dtype=torch.float64)
            full[self.bases[s]:] = q[at:at + n]
            o = (oracle.sink_attention(full, k, v, self.scale, d(self.sink)) if self.sink is not None
                 else oracle.banded_attention(full, k, v, self.scale, self.window or None))
            out.append(o[self.bases[s]:])
            at += n
        o = torch.cat(out)
        if self.gate is not None:
            o = o * torch.sigmoid(d(self.gate).view(-1, self.heads, self.vdim_p)[..., : self.vdim])
        return o


SHAPES = [(3, 20, 6, 36, 44), (1, 64, 64, 64, 64), (20, 128, 64, 128, 512), (17, 72, 2, 40, 256), (2, 8, 8, 8, 8), (16, 128, 32, 96, 200)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SHAPES)
def test_latent_norm_rotation_and_append(dtype, shape):
    """Also at positions far out, where a rounded angle would be off."""
    heads, dim, rot, vdim, rank = shape
    c = Case(dtype, *shape, lens=[5, 1, 18], bases=[0, 15, 200003], base=500.0 if heads == 1 else 1e6)
    c.prep()
    tol = 2e-6 if dtype == F32 else 8e-3
    raw, pos, T = d(c.raw), c.batch[4].cpu(), sum(c.lens)
    seq = c.batch[3].long().cpu()
    row = d(c.cache)[c.table.cpu()[seq, pos // PAGE].long(), (pos % PAGE).long(), 0]
    close(row[:, :rank], oracle.rms_norm(raw[:, c.off["c"]: c.off["c"] + rank], d(c.gamma), 1e-5), tol)
    close(row[:, c.rank_p: c.rank_p + rot], oracle.rotate_pairs(raw[:, c.off["kr"]: c.off["kr"] + rot], pos, c.base), tol)
    qr = raw[:, c.off["qr"]: c.off["c"]].view(T, heads, c.rot_p)[..., :rot]
    close(d(c.queries()[1])[..., :rot], oracle.rotate_pairs(qr, pos, c.base), tol)
    assert torch.equal(c.proj[:, : c.off["qr"]], c.raw[:, : c.off["qr"]])          # the unrotated part stays
    pads = torch.cat([row[:, rank:c.rank_p], row[:, c.rank_p + rot:]], 1)
    assert float(pads.abs().sum()) == 0.0


@pytest.mark.parametrize("how,dtype", [("any", F32), ("any", BF16), ("decode", BF16), ("prefill", BF16)])
@pytest.mark.parametrize("shape", SHAPES)
def test_latent_attention(how, dtype, shape):
    lens, bases = ([1, 1, 1, 1, 1], [0, 15, 16, 300, 63]) if how == "decode" else ([33, 2, 1, 270], [0, 15, 48, 130])
    c = Case(dtype, *shape, lens=lens, bases=bases, scale=2.0 * (shape[1] + shape[2]) ** -0.5)
    c.prep()
    want = c.want()
    for splits in ((1, 2, 5, 64) if how == "decode" else (1,)):
        close(c.run(how, splits), want, 2e-5 if dtype == F32 else 2.5e-2)


def test_wide_latents_take_the_plain_kernel():
    c = Case(BF16, 2, 24, 10, 16, 700, lens=[3, 40], bases=[70, 0])
    assert not c.lat.decode_ok(PAGE) and not c.lat.prefill_ok(136, 64)
    c.prep()
    close(c.run("any"), c.want(), 2.5e-2)


@pytest.mark.parametrize("how", ["any", "decode", "prefill"])
@pytest.mark.parametrize("sink", [-30.0, 0.0, 4.0, 200.0])
def test_sink_takes_its_share(how, sink):
    lens, bases = ([1, 1], [0, 100]) if how == "decode" else ([20, 17], [0, 90])
    c = Case(BF16, 3, 32, 16, 32, 48, lens=lens, bases=bases, sink=sink)
    c.prep()
    got, want = c.run(how, 2), c.want()
    assert float((d(got) - want).abs().max()) < 0.02 * max(0.05, float(want.abs().max()))
    if sink == 200.0:
        assert float(got.abs().max()) == 0.0


@pytest.mark.parametrize("how", ["any", "decode", "prefill"])
def test_one_key_that_stands_out_is_found_wherever_it_lies(how):
    """Key j alone matches the last query, once by its latent and once by its rotated part."""
    n, shape = 333, (2, 40, 24, 40, 64)
    for j in (0, 1, 15, 16, 17, 63, 64, 127, 128, 255, 256, 319, 320, 331, 332):
        for part in ("latent", "rotated"):
            lens, bases = ([1], [n - 1]) if how == "decode" else ([40], [n - 40])
            c = Case(BF16, *shape, lens=lens, bases=bases, seed=j, scale=1.5, sink=-5.0)
            c.prep()
            at, q, qr = int(c.table[0, j // PAGE]), *c.queries()
            row = c.cache[at, j % PAGE, 0]
            if part == "latent":
                row[: c.rank] = (q[-1, 0].float() @ c.uk[0].float()).to(BF16) * 2
            else:
                row[c.rank_p: c.rank_p + c.rot] = qr[-1, 0] * 2
            v = d(c.uv[0]) @ d(row[: c.rank])
            got = d(c.run(how, 3))[-1, 0]
            assert float((got - v).abs().max()) < 0.03 * float(v.abs().max()) + 0.02, (j, part)


def test_short_and_long_portions_in_one_batch_stay_apart():
    """Sequences below the threshold are left to the single-token form; their rows of the output are not touched."""
    c = Case(BF16, 4, 64, 32, 64, 96, lens=[3, 40, 1], bases=[20, 5, 77])
    c.prep()
    want = c.want()
    cu = torch.tensor([0, 0, 45, 45], dtype=torch.int32, device="cuda")
    lat = torch.empty(45, c.W, device="cuda", dtype=BF16)
    c.lat.gather(c.table, c.cache, cu, torch.zeros_like(cu[1:]), 45, lat)
    kv = torch.zeros(45, 4 * 128, device="cuda", dtype=BF16)
    k, v = kv[:, :256].unflatten(1, (4, 64)), kv[:, 256:].unflatten(1, (4, 64))
    k.copy_(torch.einsum("tr,hdr->thd", lat[:, :96].float(), c.uk.float()))
    v.copy_(torch.einsum("tr,hdr->thd", lat[:, :96].float(), c.uv.float()))
    out = torch.full((44, 4, 64), 7.0, device="cuda", dtype=BF16)
    c.lat.attn_prefill(c.queries()[0], c.proj, k, v, lat, c.batch, cu, c.batch[1], 40, 16, None, out, status())
    close(out[3:43], want[3:43], 2.5e-2)
    assert float((out[:3] - 7.0).abs().max()) == 0.0 and float((out[43:] - 7.0).abs().max()) == 0.0


# ------------------------------------------------------------------------------- experts
def _route(z, corr, E, top, groups, keep, tile):
    T = z.shape[0]
    i32 = dict(device="cuda", dtype=torch.int32)
    idx, slot, row = (torch.full((T, top), -1, **i32) for _ in range(3))
    weight = torch.full((T, top), float("nan"), device="cuda")
    counts, offset, count = torch.zeros(E + 1, **i32), torch.full((E,), -1, **i32), torch.full((1,), -1, **i32)
    tiles = torch.full((min(T * top, E + T * top // tile), 3), -1, **i32)
    plan = (idx, weight, slot, counts, offset, tiles, count)
    H().expert_select(z, corr, (E, top, groups, keep), tile, *plan)
    return plan, row


@pytest.mark.parametrize("E,top,groups,keep,T", [(12, 3, 4, 2, 50), (1, 1, 1, 1, 3), (64, 6, 8, 3, 300), (100, 7, 5, 5, 33), (8, 8, 2, 2, 9),
                                                 (256, 8, 8, 4, 1), (40, 1, 40, 1, 70), (512, 32, 1, 1, 17)])
def test_expert_choice(E, top, groups, keep, T):
    """Choice scores of both signs (a masked group must lose against a negative score), weights without correction."""
    g = torch.Generator().manual_seed(E + T)
    z = torch.randn(T, E, generator=g) * 2
    corr = torch.randn(E, generator=g) * 0.5 - 0.6          # most choice scores are negative
    zc, cc = z.cuda(), corr.cuda()
    for tile in (16, 128):
        (idx, weight, slot, counts, offset, tiles, count), _ = _route(zc, cc, E, top, groups, keep, tile)
        r = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
        per = [0] * E
        for t in range(T):
            want = oracle.choose_experts(z[t].double(), corr.double(), r)
            got = dict(zip(idx[t].tolist(), weight[t].tolist()))
            assert sorted(got) == sorted(e for e, _ in want)
            assert all(abs(got[e] - float(w)) < 1e-6 for e, w in want)
            for e in got:
                per[e] += 1
        # segments in order, every place once, tiles cover them
        off = offset.tolist()
        assert off == [sum(per[:e]) for e in range(E)]
        places = (offset[idx.long()] + slot).flatten()
        assert sorted(places.tolist()) == list(range(T * top))
        tl = tiles[: int(count)].tolist()
        assert [(e, a, n) for e, a, n in tl] == [(e, off[e] + r0, min(tile, per[e] - r0)) for e in range(E) for r0 in range(0, per[e], tile)]
        assert int(counts.abs().sum()) == 0


@pytest.mark.parametrize("dtype,tile", [(F32, 64), (BF16, 16), (BF16, 32), (BF16, 64), (BF16, 128)])
@pytest.mark.parametrize("T,E,top,dim,ff,limit", [(3, 4, 2, 72, 24, 0.5), (150, 6, 3, 136, 40, 1.0), (700, 3, 2, 320, 136, 6.0)])
def test_experts_of_a_batch(dtype, tile, T, E, top, dim, ff, limit):
    """Rows gathered by expert, both grouped products, weighted sum with norm and residual; expert 0 is never chosen."""
    g = torch.Generator().manual_seed(T)
    C, c = H(), lambda t: t.to("cuda", dtype)
    h, z = c(torch.randn(T, dim, generator=g)), torch.randn(T, E, generator=g).cuda()
    z[:, 0] -= 50
    w_in, w_out = c(torch.randn(E, 2 * ff, dim, generator=g) * 2 * dim ** -0.5), c(torch.randn(E, dim, ff, generator=g) * ff ** -0.5)
    plan, row = _route(z, torch.zeros(E, device="cuda"), E, top, 1, 1, tile)
    idx, weight, slot, counts, offset, tiles, count = plan
    n, act = T * top, (2, limit, 1.702)
    x, a, y = (torch.full((n, k), float("nan"), device="cuda", dtype=dtype) for k in (dim, ff, dim))
    C.expert_gather(h, (E, top, 1, 1), *plan, x, row)
    assert torch.equal(x[row.flatten().long()], h.repeat_interleave(top, 0))
    if dtype == F32:
        gu = torch.empty(n, 2 * ff, device="cuda")
        C.gemm_tiles(x, w_in, gu, tiles, count, tile, 0, 0, act, status())
        C.gate_pair(gu, ff, ff, act, a)
    else:
        C.gemm_tiles(x, w_in, a, tiles, count, tile, ff, ff, act, status())
    C.gemm_tiles(a, w_out, y, tiles, count, tile, 0, 0, act, status())
    tol = 1e-5 if dtype == F32 else 2e-2
    W = {}
    for e in range(E):
        W.update({f"e{e}.gate": d(w_in[e, :ff]), f"e{e}.up": d(w_in[e, ff:]), f"e{e}.down": d(w_out[e])})
    want = torch.zeros(n, dim, dtype=torch.float64)
    rc, ic, hd = row.cpu(), idx.cpu(), d(h)
    for e in range(E):
        t, j = (ic == e).nonzero(as_tuple=True)
        if t.numel():
            want[rc[t, j].long()] = oracle.clamped_expert(hd[t], W, f"e{e}.", limit)
    close(y, want, tol)
    out, xs = torch.empty(T, dim, device="cuda", dtype=dtype), torch.randn(T, dim, device="cuda")
    wp, x0 = 1 + 0.3 * torch.randn(dim, device="cuda"), d(xs)
    C.expert_norm(y, None, row, weight, wp, xs, None, out, 1e-4, 0.7)
    total = (d(y)[rc.long()] * d(weight)[..., None]).sum(1)
    ref = x0 + 0.7 * oracle.rms_norm(total, d(wp), 1e-4)
    close(xs, ref, 1e-5)
    close(out, ref, 1e-5 if dtype == F32 else 5e-3)


@pytest.mark.parametrize("act,fn", [((1, 0.0, 0.0), lambda g, u: torch.clamp(g, min=0) * u),
                                    ((2, 0.8, 1.702), lambda g, u: torch.clamp(g, max=0.8) * torch.sigmoid(1.702 * torch.clamp(g, max=0.8))
                                     * (torch.clamp(u, -0.8, 0.8) + 1))])
def test_gated_activations(act, fn):
    g = torch.Generator().manual_seed(1)
    gu = torch.randn(37, 104, generator=g).cuda()
    out = torch.full((37, 48), float("nan"), device="cuda")
    H().gate_pair(gu, 41, 56, act, out)
    close(out[:, :41], fn(d(gu)[:, :41], d(gu)[:, 56:97]), 1e-6)
    assert float(out[:, 41:].abs().sum()) == 0.0
    x, w = torch.randn(9, 64, generator=g).to("cuda", BF16), torch.randn(88, 64, generator=g).to("cuda", BF16) / 8
    y = torch.empty(9, 40, device="cuda", dtype=BF16)
    H().gemm_decode(x, w, y, 40, 48, 1.0, status(), act)
    p = d(x) @ d(w).t()
    close(y, fn(p[:, :40], p[:, 48:]), 1e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,b,N,K", [(1, 16, 512, 128), (7, 3, 44, 24), (150, 5, 136, 72), (64, 1, 8, 8)])
def test_products_per_head(dtype, rows, b, N, K):
    g = torch.Generator().manual_seed(N)
    wide = torch.randn(rows, b * K + 24, generator=g).to("cuda", dtype)            # heads inside a wider row
    w = torch.randn(b, N, K, generator=g).to("cuda", dtype)
    x = wide[:, 8: 8 + b * K].unflatten(1, (b, K))
    out = torch.full((rows, b, N), float("nan"), device="cuda", dtype=dtype)
    H().gemm_heads(x, w, out, status())
    close(out, torch.einsum("tbk,bnk->tbn", d(x), d(w)), 1e-5 if dtype == F32 else 6e-3)


# ------------------------------------------------------------------------------- norms and token input
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim", [100, 333, 2048])
def test_norm_on_the_output_only(dtype, dim):
    torch.manual_seed(dim)
    y = (torch.randn(6, dim, device="cuda") * 3).to(dtype)
    w, x = 1 + 0.3 * torch.randn(dim, device="cuda"), torch.randn(6, dim, device="cuda")
    x0 = d(x)
    h = torch.full((6, pad8(dim)), float("nan"), device="cuda", dtype=dtype)
    H().sandwich_norm(y, None, None, None, w, x, None, h, 1e-2, 0.3)
    want = x0 + 0.3 * oracle.rms_norm(d(y), d(w), 1e-2)
    close(x, want, 1e-6)
    close(h[:, :dim], want, 1e-6 if dtype == F32 else 5e-3)
    assert float(h[:, dim:].float().abs().sum()) == 0.0
    emb, ids = torch.randn(50, dim, device="cuda").to(dtype), torch.tensor([3, 49, 0, 3, 7, 1], device="cuda", dtype=torch.int32)
    H().embed_pos_norm(ids, ids, emb, None, 1.0, None, x, h, 1e-5)
    close(x, d(emb)[ids.long().cpu()], 1e-9)
    close(h[:, :dim], d(emb)[ids.long().cpu()], 1e-9)


@pytest.mark.parametrize("rows,dim,n", [(1, 64, 16), (9, 104, 8), (200, 320, 136)])
def test_token_input(rows, dim, n):
    g = torch.Generator().manual_seed(rows)
    table = torch.randn(30, 3 * n, generator=g)
    ids = torch.randint(0, 30, (rows,), generator=g, dtype=torch.int32).cuda()
    x, w = torch.randn(rows, dim, generator=g), torch.randn(n, dim, generator=g) * 2 * dim ** -0.5
    for dtype, tol in ((F32, 1e-5), (BF16, 1e-2)):
        t, xx, ww = (v.to("cuda", dtype) for v in (table, x, w))
        part = t[:, n: 2 * n]                               # the middle layer's share
        want = oracle.gelu_tanh(d(xx) @ d(ww).t()) * d(part)[ids.long().cpu()]
        out = torch.empty(rows, n, device="cuda", dtype=dtype)
        if dtype == BF16:
            H().gemm_decode(xx, ww, out, 0, 0, 1.0, status(), (0, 0.0, 0.0), part, ids)
            close(out, want, tol)
        H().gemm_nt(xx, ww, out, 1.0, status())
        H().gelu_mul(out, part, ids)
        close(out, want, tol)


# ------------------------------------------------------------------------------- engine
def test_prefixes_are_shared_where_pages_determine_everything():
    cfg = hu.CONFIGS["latent_ragged"]
    w, toks = hu.weights(cfg, 3), hu.tokens(cfg, 70)
    want = oracle.forward(cfg, w, toks)
    eng = engine(cfg, "float32", w=w)
    a, la = eng.start_sequence(toks[:60])
    b, lb = eng.start_sequence(toks)
    assert eng.last_prefix_hit == 48 and hu.rel(la, want[59:60]) < 5e-5 and hu.rel(lb, want[69:70]) < 5e-5
    eng.release(a)
    eng.release(b)
    assert eng.cache.alloc.used == 0


def test_batch_and_portions_do_not_change_32_bit_logits_beyond_rounding():
    """One request alone, beside others, and cut into portions of two tokens."""
    cfg = hu.CONFIGS["latent_wide"]
    w, toks = hu.weights(cfg, 12), hu.tokens(cfg, 64, 5)
    eng = engine(cfg, "float32", w=w)
    s = eng.cache.new_sequence()
    alone = eng.step([s], [toks], [list(range(64))])
    eng.release(s)
    s, o = eng.cache.new_sequence(), eng.cache.new_sequence()
    beside = eng.step([o, s], [hu.tokens(cfg, 90, 6), toks], [[], list(range(64))])
    eng.release(s)
    s, out = eng.cache.new_sequence(), []
    for i in range(0, 64, 2):
        lists = [toks[i:i + 2]] if i % 3 else [toks[i:i + 2], [i]]
        out.append(eng.step([s] if i % 3 else [s, o], lists, [[0, 1], []][: len(lists)]))
    for other in (beside, torch.cat(out)):
        assert hu.rel(other, alone) < 2e-5

"""Layer-list models without a GPU: configuration, registry, checkpoint folders, caches with unequal key
and value widths, request handling of the trace replay, and the sensitivity of the oracle."""
import json
import os

import pytest
import torch

import hybrid_oracle as oracle
import hybrid_util as hu
from mythos_b200.infer.kv_paged import PagedKVCache, RecurrentStatePool
from mythos_b200.models import registry
from mythos_b200.models.hybrid import HybridModel, expected_shapes
from mythos_b200.models.hybrid_config import (FrequencyScaling, HybridConfig, RampScaling, Rotation, dogozen_config, lebedra_config,
                                               teganex_config, zigivik_config)
from mythos_b200.oil.importers import read_safetensors_torch, write_safetensors
from mythos_b200.oil.model_io import load_model


@pytest.mark.parametrize("name", sorted(hu.CONFIGS))
def test_config_round_trip(name):
    cfg = HybridConfig.from_dict(hu.CONFIGS[name])
    assert cfg.to_dict() == hu.CONFIGS[name]
    assert HybridConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"].update(heads=0),
    lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c.update(architecture="Unheard"),
    lambda c: c["layers"][0].update(type="latent_attention"),
])
def test_bad_configurations_are_refused(tmp_path, change):
    raw = json.loads(json.dumps(hu.CONFIGS["ragged"]))
    change(raw)
    (tmp_path / "config.json").write_text(json.dumps(raw))
    with pytest.raises((ValueError, KeyError)):
        registry.load_config(str(tmp_path))


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0]["mixer"].update(rot_dim=7, rot={"base": 10.0, "dims": 7}),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=5),
    lambda c: c["layers"][1]["mlp"].update(kind="other"),
    lambda c: c["layers"][0].update(type="gla"),
])
def test_bad_latent_configurations_are_refused(change):
    raw = json.loads(json.dumps(hu.CONFIGS["latent_ragged"]))
    change(raw)
    with pytest.raises((ValueError, KeyError)):
        HybridConfig.from_dict(raw)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][2]["mixer"].update(kv_from=1),            # other widths
    lambda c: c["layers"][2]["mixer"].update(kv_from=2),
    lambda c: c["layers"][0]["mixer"].update(kv_from=2),            # a later layer
    lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=9),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=22),
    lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=-1),
    lambda c: c["layers"][1]["mixer"]["right"].update(state=0),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4),
    lambda c: c["layers"][1]["mlp"].update(kind="other"),
    lambda c: c["layers"][1].update(type="gla"),
])
def test_bad_scan_configurations_are_refused(change):
    raw = json.loads(json.dumps(hu.CONFIGS["scan_ragged"]))
    change(raw)
    with pytest.raises((ValueError, KeyError)):
        HybridConfig.from_dict(raw)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][2]["mixer"].update(kv_from=1),            # not latents
    lambda c: c["layers"][2]["mixer"].update(kv_from=2),
    lambda c: c["layers"][2]["mixer"].update(kv_rank=40),
    lambda c: c["layers"][2]["mixer"]["rot"].update(base=301.0),    # rotated otherwise than the latents it uses
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4),
    lambda c: c["layers"][0]["mixer"].update(q_rank=0),
    lambda c: c["layers"][1]["mixer"].update(vdim=24),              # the keys are the values
    lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][1]["mlp"].update(kind="moe"),
    lambda c: c["layers"][3].update(type="parallel"),
    lambda c: c["canon"].update(taps=-1),
])
def test_bad_parallel_configurations_are_refused(change):
    raw = json.loads(json.dumps(hu.CONFIGS["side_ragged"]))
    change(raw)
    with pytest.raises((ValueError, KeyError)):
        HybridConfig.from_dict(raw)


def test_shapes_of_parallel_sublayers():
    raw = json.loads(json.dumps(hu.CONFIGS["side_ragged"]))
    del raw["layers"][2]["mixer"]["mask"]
    c = HybridConfig.from_dict(raw)
    shapes = expected_shapes(c)
    assert c.layers[2].mixer.window == 0 and c.layers[2].mixer.rotation == c.layers[0].mixer.rotation
    assert shapes["embed.norm"] == shapes["l2.norm1"] == shapes["final.norm"] == () and shapes["l3.canon1"] == (100, 3)
    for absent in ("l0.norm2", "l0.norm1b", "l1.mix.v", "l1.mix.sink", "l2.mix.dkv", "l2.mix.dkv.norm", "l2.mlp.up", "l0.mix.q", "l1.mlp.gate"):
        assert absent not in shapes
    assert shapes["l2.mix.uq"] == (5 * 18, 21) and shapes["l1.mlp.act"] == (4,) and shapes["l1.mix.k.b"] == (40,)


def test_optional_parts_of_a_configuration():
    raw = json.loads(json.dumps(hu.CONFIGS["scan_ragged"]))
    del raw["layers"][0]["mixer"]["q_temp"], raw["layers"][1]["mixer"]["left"]["mask"], raw["layers"][1]["mlp"]["router"]["groups"]
    raw["layers"][1]["mlp"]["shared"], raw["logit_softcap"], raw["layers"][0]["mlp"] = None, None, None
    c = HybridConfig.from_dict(raw)
    left, moe = c.layers[1].mixer.left, c.layers[1].mlp
    assert c.layers[0].mixer.q_temp is None and left.window == 0 and (moe.groups, moe.keep, moe.shared) == (1, 1, 0)
    assert c.logit_softcap == 0.0 and c.layers[0].mlp is None
    shapes = expected_shapes(c)
    assert "l1.mlp.shared.gate" not in shapes and "l2.mix.k" not in shapes and "l2.mix.v.b" not in shapes and "l0.mix.k.b" in shapes


@pytest.mark.parametrize("rot", [{"base": 1e4, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}},
                                 {"base": 500.0, "dims": 10}, {"base": 1e5, "dims": 48, "scaling": {"factor": 2.0, "low": 2.0, "high": 2.0, "original": 64}}])
def test_rotation_frequencies(rot):
    sc = rot.get("scaling")
    r = Rotation(rot["base"], rot["dims"], FrequencyScaling(**sc) if sc else None)
    want = torch.tensor(oracle.frequencies(rot), dtype=torch.float64) / (2 * torch.pi)
    assert torch.allclose(torch.tensor(r.turns(), dtype=torch.float64), want, rtol=1e-12, atol=0)


@pytest.mark.parametrize("rot", [hu.ramp(1e4, 64, 8.0, 256, 32.0), hu.ramp(500.0, 10, 2.5, 4096, 32.0), hu.ramp(300.0, 6, 4.0, 64, 3.0, 3.0),
                                 hu.ramp(100.0, 2, 16.0, 16, 4.0, 0.5), hu.ramp(1e5, 48), hu.ramp(10.0, 16, 1.0, 32, 4.0)])
def test_ramped_rotation_frequencies(rot):
    sc = rot.get("scaling")
    r = Rotation(rot["base"], rot["dims"], RampScaling(**sc) if sc else None)
    freq, amp = oracle.yarn_frequencies(rot)
    want = torch.tensor(freq, dtype=torch.float64) / (2 * torch.pi)
    assert torch.allclose(torch.tensor(r.turns(), dtype=torch.float64), want, rtol=1e-12, atol=0) and r.amplitude == pytest.approx(amp, rel=1e-12)


def _write(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), w)


def test_checkpoint_folder_loads_through_the_registry(tmp_path):
    cfg = hu.CONFIGS["ragged"]
    w = hu.weights(cfg, 3)
    w["table"] = torch.arange(5, dtype=torch.int32)
    _write(str(tmp_path), cfg, w)
    back = read_safetensors_torch(str(tmp_path / "model.safetensors"))
    assert all(back[n].dtype == t.dtype and torch.equal(back[n], t) for n, t in w.items())
    m, rd = load_model(str(tmp_path))
    assert rd is None and isinstance(m, HybridModel) and m.cfg.num_layers == len(cfg["layers"])
    assert torch.equal(m.tensor("l1.mix.right.q.conv"), w["l1.mix.right.q.conv"])
    with pytest.raises(RuntimeError):
        m(torch.zeros(1, 4, dtype=torch.int32))           # no CPU forward
    from mythos_b200.infer.server import ModelZoo

    assert ModelZoo(str(tmp_path.parent)).scan()[tmp_path.name] == str(tmp_path)
    from mythos_b200.tools.info import main as info_main

    assert info_main([str(tmp_path)]) == 0


def test_lebedra_folder_loads_through_the_registry(tmp_path):
    cfg = hu.CONFIGS["latent_ragged"]
    w = hu.weights(cfg, 3)
    _write(str(tmp_path), cfg, w)
    m, _ = load_model(str(tmp_path))
    assert isinstance(m, HybridModel) and m.cfg.architecture == "Lebedra" and not m.cfg.pre_norm
    assert torch.equal(m.tensor("l1.mlp.e5.down"), w["l1.mlp.e5.down"]) and torch.equal(m.tensor("l0.mix.sink"), w["l0.mix.sink"])
    assert m.cfg.context_limit > m.cfg.max_seq_len and "l2.norm2" not in dict(m.named_tensors())
    del w["l1.mlp.correction"]
    with pytest.raises(KeyError):
        HybridModel(HybridConfig.from_dict(cfg), w)


def test_dogozen_folder_loads_through_the_registry(tmp_path):
    cfg = hu.CONFIGS["scan_ragged"]
    w = hu.weights(cfg, 3)
    _write(str(tmp_path), cfg, w)
    m, _ = load_model(str(tmp_path))
    assert isinstance(m, HybridModel) and m.cfg.architecture == "Dogozen" and m.cfg.tied_head and m.cfg.norm_offset == 1.0
    assert torch.equal(m.tensor("l1.mix.right.A_log"), w["l1.mix.right.A_log"]) and "head" not in dict(m.named_tensors())
    from mythos_b200.tools.info import main as info_main

    assert info_main([str(tmp_path)]) == 0
    del w["l1.mix.left.sink"]
    with pytest.raises(KeyError):
        HybridModel(HybridConfig.from_dict(cfg), w)


def test_zigivik_folder_loads_through_the_registry(tmp_path):
    cfg = hu.CONFIGS["side_ragged"]
    w = hu.weights(cfg, 3)
    _write(str(tmp_path), cfg, w)
    m, _ = load_model(str(tmp_path))
    assert isinstance(m, HybridModel) and m.cfg.architecture == "Zigivik" and m.cfg.parallel and m.cfg.input_conv == 3
    assert m.tensor("embed.norm").shape == () and torch.equal(m.tensor("l2.mix.uk"), w["l2.mix.uk"])
    from mythos_b200.tools.info import main as info_main

    assert info_main([str(tmp_path)]) == 0
    del w["l1.mlp.act"]
    with pytest.raises(KeyError):
        HybridModel(HybridConfig.from_dict(cfg), w)


def test_missing_and_misshapen_tensors_are_refused():
    cfg = hu.CONFIGS["single"]
    hc = HybridConfig.from_dict(cfg)
    w = hu.weights(cfg)
    short = {k: v for k, v in w.items() if k != "l1.mix.a2.b"}
    with pytest.raises(KeyError):
        HybridModel(hc, short)
    w["l0.mlp.down"] = w["l0.mlp.down"][:, :-1]
    with pytest.raises(ValueError):
        HybridModel(hc, w)


def test_named_configuration_has_consistent_shapes():
    cfg = teganex_config(width=256, layers=4, vocab=64, max_positions=32)
    m = HybridModel.random(cfg, low_rank=8)
    assert m.param_count() == sum(t.numel() for _, t in m.named_tensors())
    assert [s.type for s in cfg.layers] == ["gla", "gla", "gla", "parallel"]
    m = HybridModel.random(dogozen_config(width=256, layers=6, vocab=64, experts=16, top=2))
    assert m.param_count() == sum(t.numel() for _, t in m.named_tensors()) and m.cfg.layers[4].mixer.kv_from == 2
    m = HybridModel.random(zigivik_config(width=512, layers=5, vocab=64))
    assert m.param_count() == sum(t.numel() for _, t in m.named_tensors()) and m.cfg.layers[1].mixer.kv_from == 0
    m = HybridModel.random(lebedra_config(width=256, layers=2, vocab=64, experts=8, top=2))
    assert m.param_count() == sum(t.numel() for _, t in m.named_tensors()) and m.tensor("l1.mlp.e7.gate").shape[1] == 256


def test_cache_with_unequal_widths_and_state_slots():
    states = RecurrentStatePool(3, "cpu")
    s0 = states.add(2, 4, 5)
    c = PagedKVCache(2, 0, 0, num_pages=6, page_size=4, max_seqs=3, max_pages_per_seq=4, device="cpu",
                     layer_shapes=[(1, 8, 16), (2, 4, 8)], states=states)
    assert c.k[0].shape == (6, 4, 1, 8) and c.v[1].shape == (6, 4, 2, 8)
    a = c.new_sequence()
    c.reserve(a, 9)
    c.advance(a, 9)
    c.k[1][int(c.block_table_host[a, 2]), 0] = 7.0
    s0[a] = 3.0
    toks = list(range(9))
    c.publish_prefix(a, toks)
    b = c.new_sequence()
    assert c.share_prefix(b, toks) == 0                    # pages alone do not determine the states
    c.free_sequence(b)
    h = c.offload_sequence(a)
    assert c.alloc.used == 0
    s0.zero_()
    other = c.new_sequence()
    a2 = c.restore_sequence(h)
    assert a2 != other and c.lens[a2] == 9 and float(s0[a2].min()) == 3.0
    assert float(c.k[1][int(c.block_table_host[a2, 2]), 0].min()) == 7.0
    assert c.size_bytes() == sum(t.numel() * 2 for t in c.k + c.v) + s0.numel() * 4


def test_pages_of_rows_without_separate_values():
    c = PagedKVCache(2, 0, 0, num_pages=5, page_size=4, max_seqs=2, max_pages_per_seq=4, device="cpu",
                     layer_shapes=[(1, 24, 0), (1, 16, 0)])
    assert c.k[0].shape == (5, 4, 1, 24) and c.v[0].numel() == 0 and c.size_bytes() == 5 * 4 * 40 * 2
    a = c.new_sequence()
    c.reserve(a, 6)
    c.advance(a, 6)
    c.k[1][int(c.block_table_host[a, 1]), 1] = 3.0
    b = c.restore_sequence(c.offload_sequence(a))
    assert c.lens[b] == 6 and float(c.k[1][int(c.block_table_host[b, 1]), 1].min()) == 3.0
    c.publish_prefix(b, list(range(6)))
    other = c.new_sequence()
    assert c.share_prefix(other, list(range(9))) == 4      # pages alone determine such a prefix


def test_batch_plan_separates_long_and_short_portions():
    from mythos_b200.infer.hybrid import EXPAND_TOKENS, HybridEngine

    class Cfg:
        cfg = HybridConfig.from_dict(hu.CONFIGS["latent_ragged"])

    n = EXPAND_TOKENS
    assert HybridEngine._batch_plan(Cfg, [1, n - 1], [5, 0]) == ([], None)
    lists, build = HybridEngine._batch_plan(Cfg, [2, n, 1, n + 3], [7, 0, 0, 100])
    assert lists == [[0, 0, n, n, 2 * n + 103], [0] * 4, [9, n, 1, n + 103], [0, 1, n + 2], [0, 0, 2], [7, 8, 0]]
    sp = build(*[torch.tensor(x, dtype=torch.int32) for x in lists])
    assert sp.keys == 2 * n + 103 and sp.max_k == n + 103 and sp.short.dtype == torch.int64
    lists, build = HybridEngine._batch_plan(Cfg, [n], [3])
    assert lists == [[0, n + 3], [0], [n + 3], [], [], []] and build(*[torch.tensor(x) for x in lists]).short is None


def test_batch_plan_leaves_out_what_no_window_reaches():
    from mythos_b200.infer.hybrid import EXPAND_TOKENS, HybridEngine

    class Cfg:
        cfg = HybridConfig.from_dict(hu.CONFIGS["side_ragged"])          # windows of 19 and 33

    n = EXPAND_TOKENS
    lists, build = HybridEngine._batch_plan(Cfg, [n, 2, n + 5], [100, 90, 32])
    assert lists == [[0, n + 32, n + 32, 2 * n + 69], [68, 0, 0], [n + 32, 92, n + 37], [n, n + 1], [1, 1], [90, 91]]
    assert build(*[torch.tensor(x, dtype=torch.int32) for x in lists]).max_k == n + 37
    Cfg.cfg.layers[0].mixer.window = 0                                   # a layer that sees everything
    assert HybridEngine._batch_plan(Cfg, [n], [100])[0][:3] == [[0, n + 100], [0], [n + 100]]


class _FakeEngine:
    """Counts tokens of every sequence; the logits of a place are its position."""

    def __init__(self, slots=2, pages=8):
        self.cache = PagedKVCache(1, 1, 1, pages, 4, slots, pages, device="cpu")
        self.max_batch = slots
        self.batches = []

    def step(self, seqs, lists, want=None):
        c = self.cache
        out = []
        self.batches.append([len(t) for t in lists])
        want = want if want is not None else [[len(t) - 1] for t in lists]
        for s, t, w in zip(seqs, lists, want):
            c.reserve(s, len(t))
            for p in w:
                row = torch.zeros(16)
                row[(c.lens[s] + p) % 16] = 1.0
                out.append(row)
            c.advance(s, len(t))
        return torch.stack(out) if out else None

    def release(self, s):
        self.cache.free_sequence(s)


def test_trace_replay_admits_continues_and_releases():
    from mythos_b200.tools.trace_run import TraceReplay

    eng = _FakeEngine()
    r = TraceReplay(eng)
    out = r.run({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [0, 2]},
                                        {"id": "b", "tokens": [4], "want": []}], "end": []})
    assert out.argmax(-1).tolist() == [0, 2]
    assert r.run({"step": 1, "entries": [{"id": "b", "tokens": [5, 6], "want": []}], "end": ["b"]}) is None
    out = r.run({"step": 2, "entries": [{"id": "c", "tokens": [9, 9], "want": [1]}, {"id": "a", "tokens": [7], "want": [0]}],
                 "end": ["a", "c"]})
    assert out.argmax(-1).tolist() == [1, 3] and eng.cache.alloc.used == 0 and not any(eng.cache.active)


def test_batcher_mixes_portions_with_decoded_tokens():
    from mythos_b200.infer.serving import ContinuousBatcher

    eng = _FakeEngine(slots=2, pages=8)
    cb = ContinuousBatcher(eng, chunk_tokens=4)
    reqs = [cb.submit([1] * n, max_new_tokens=3) for n in (2, 11, 5)]
    done = cb.run_until_idle()
    assert len(done) == 3 and eng.cache.alloc.used == 0
    for r, n in zip(reqs, (2, 11, 5)):
        assert r.output == [n - 1, n, n + 1]               # logits named the positions n - 1, n, n + 1
    assert any(1 in b and max(b) > 1 for b in eng.batches)  # a decoded token beside a portion
    assert max(sum(b) for b in eng.batches) <= 5
    with pytest.raises(MemoryError):
        cb.submit([1] * 100)
        cb.run_until_idle()


# ------------------------------------------------------------------ the oracle notices mistakes
def _slip(name):
    """A copy of one mechanism with a mistake in it."""
    def late_write(q, k, v, g, beta):                      # read-out before the current token's write
        T, H, dk = q.shape
        S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype)
        out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = g[t][:, :, None] * S
            out[t] = torch.einsum("hkv,hk->hv", S, q[t])
            u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
        return out

    def no_decay(q, k, v, alpha):
        return oracle_gla(q, k, v, torch.ones_like(alpha))

    def shifted_conv(x, w):
        return oracle_conv(torch.cat([torch.zeros_like(x[:1]), x[:-1]]), w)

    def blind(q, k, v, scale):                             # the newest key is left out
        T = q.shape[0]
        keep = oracle_att(q[:-1], k[:-1], v[:-1], scale)
        return torch.cat([v[:1].repeat_interleave(q.shape[1] // v.shape[1], 1), keep[: T - 1]])

    return {"late_write": ("delta_recurrence", late_write), "no_decay": ("gla_recurrence", no_decay),
            "shifted_conv": ("short_conv", shifted_conv), "blind": ("causal_attention", blind)}[name]


oracle_gla, oracle_conv, oracle_att = oracle.gla_recurrence, oracle.short_conv, oracle.causal_attention


@pytest.mark.parametrize("slip", ["late_write", "no_decay", "shifted_conv", "blind"])
def test_a_mistake_in_a_mechanism_is_larger_than_the_tolerance(slip, monkeypatch):
    cfg = hu.CONFIGS["ragged"]
    w, toks = hu.weights(cfg, 5), hu.tokens(cfg, 24)
    right = oracle.forward(cfg, w, toks)
    fn, wrong = _slip(slip)
    monkeypatch.setattr(oracle, fn, wrong)
    assert hu.rel(oracle.forward(cfg, w, toks), right) > 0.15   # bf16 comparisons allow 0.06


def _latent_slips():
    """Mistakes in Lebedra's mechanisms: name -> (function of the oracle, wrong version)."""
    att, rot, choose, expert, side, norm = (oracle.sink_attention, oracle.rotate_pairs, oracle.choose_experts, oracle.clamped_expert,
                                            oracle.token_side, oracle.rms_norm)

    def half_split(x, pos, base):
        n = x.shape[-1]
        order = torch.tensor([i // 2 + (i % 2) * (n // 2) for i in range(n)])
        out = torch.empty_like(x)
        out[..., order] = rot(x[..., order], pos, base)
        return out

    def renormalised(z, c, r, *_):
        p = choose(z, c, r)
        total = sum(w for _, w in p)
        return [(e, w / total) for e, w in p]

    def zero_mask(z, c, r, *_):                                 # other groups count as zero instead of never
        E, n, keep = r["experts"], r["groups"]["count"], r["groups"]["keep"]
        s = torch.softmax(z, -1)
        choice, size = s + c, E // n
        best = torch.topk(choice.view(n, size).amax(1), keep).indices
        ok = torch.zeros(n, dtype=torch.bool)
        ok[best] = True
        masked = torch.where(ok.repeat_interleave(size), choice, torch.zeros_like(choice))
        return [(int(e), s[e]) for e in torch.topk(masked, r["top"]).indices]

    def groups_by_sum(z, c, r, *_):
        E, n, keep = r["experts"], r["groups"]["count"], r["groups"]["keep"]
        s = torch.softmax(z, -1)
        choice, size = s + c, E // n
        best = torch.topk(choice.view(n, size).sum(1), keep).indices.tolist()
        allowed = [e for e in range(E) if e // size in best]
        return [(e, s[e]) for e in sorted(allowed, key=lambda e: -float(choice[e]))[: r["top"]]]

    return {"no_sink": ("sink_attention", lambda q, k, v, sc, sink: att(q, k, v, sc, torch.full_like(sink, -1e9))),
            "scaled_sink": ("sink_attention", lambda q, k, v, sc, sink: att(q, k, v, sc, sink * sc)),
            "no_rotation": ("rotate_pairs", lambda x, pos, base: x),
            "half_split": ("rotate_pairs", half_split),
            "late_positions": ("rotate_pairs", lambda x, pos, base: rot(x, pos if x.dim() == 3 else pos + 1, base)),
            "renormalised": ("choose_experts", renormalised),
            "weights_with_correction": ("choose_experts", lambda z, c, r, *_: [(e, w + c[e]) for e, w in choose(z, c, r)]),
            "no_correction": ("choose_experts", lambda z, c, r, *_: choose(z, torch.zeros_like(c), r)),
            "no_groups": ("choose_experts", lambda z, c, r, *_: choose(z, c, {**r, "groups": {"count": 1, "keep": 1}})),
            "groups_by_sum": ("choose_experts", groups_by_sum), "zero_mask": ("choose_experts", zero_mask),
            "no_limit": ("clamped_expert", lambda h, W, p, limit: expert(h, W, p, 1e9)),
            "no_token_input": ("token_side", lambda x, W, p, e, eps: side(x, W, p, e, eps) * 0)}


@pytest.mark.parametrize("slip", sorted(_latent_slips()))
def test_a_mistake_in_a_latent_or_expert_mechanism_shows(slip, monkeypatch):
    """Far above what 32-bit comparisons allow (5e-5), and on most rows above the bf16 tolerance as well."""
    cfg = json.loads(json.dumps(hu.CONFIGS["latent_ragged"]))
    cfg["layers"][1]["mlp"] = hu.moe(12, 3, 20, 0.7, 3, 1)
    cfg["norm"]["eps"] = 0.05                               # the scale of a sublayer's output shows
    w, toks = hu.weights(cfg, 5), hu.tokens(cfg, 40)
    w["l1.mlp.correction"] = (w["l1.mlp.correction"].float() - 0.5).to(torch.bfloat16)      # negative choice scores
    right = oracle.forward(cfg, w, toks)
    fn, wrong = _latent_slips()[slip]
    monkeypatch.setattr(oracle, fn, wrong)
    e = hu.row_errors(oracle.forward(cfg, w, toks), right)
    assert float(e.max()) > 0.06 and float((e > 1e-3).double().mean()) > 0.3, (float(e.max()), float(e.median()))


def _scan_slips():
    """Mistakes in Dogozen's mechanisms: name -> (function of the oracle, wrong version)."""
    att, rot, freq, temp, scan, choose, cap, conv, norm, soft, shared = (
        oracle.window_sink_attention, oracle.rotate_halves, oracle.frequencies, oracle.query_temperature, oracle.selective_scan,
        oracle.choose_by_sigmoid, oracle.soft_cap, oracle.short_conv, oracle.rms_norm_around_zero, oracle.softplus, oracle.tempered_attention)

    def interleaved(x, pos, r):
        n = r["dims"]
        order = torch.tensor([2 * i for i in range(n // 2)] + [2 * i + 1 for i in range(n // 2)] + list(range(n, x.shape[-1])))
        out = torch.empty_like(x)
        out[..., order] = rot(x[..., order], pos, r)
        return out

    def late_read(x, dt, A, B, C, D):                      # read-out before the current token's write
        S, out = torch.zeros_like(A), torch.zeros_like(x)
        for t in range(x.shape[0]):
            S = torch.exp(dt[t][:, None] * A) * S
            out[t] = S @ C[t] + D * x[t]
            S = S + (dt[t] * x[t])[:, None] * B[t][None, :]
        return out

    def one_best(z, r):                                    # groups by their best expert alone
        s, g = torch.sigmoid(z), r["groups"]
        size = r["experts"] // g["count"]
        best = torch.topk(s.view(g["count"], size).amax(1), g["keep"]).indices.tolist()
        picked = sorted((e for e in range(r["experts"]) if e // size in best), key=lambda e: -float(s[e]))[: r["top"]]
        total = sum(s[e] for e in picked)
        return [(e, s[e] / total * r["scale"]) for e in picked]

    def own_keys(h, W, p, c, eps, kv):                     # a sharing layer whose queries meet the previous layer's stream
        return shared(h, W, p, {k: v for k, v in c.items() if k != "q_temp"}, eps, kv)

    return {"window_longer": ("window_sink_attention", lambda q, k, v, sc, w=None, s=None: att(q, k, v, sc, w and w + 1, s)),
            "window_shorter": ("window_sink_attention", lambda q, k, v, sc, w=None, s=None: att(q, k, v, sc, w and w - 1, s)),
            "no_sink": ("window_sink_attention", lambda q, k, v, sc, w=None, s=None: att(q, k, v, sc, w)),
            "scaled_sink": ("window_sink_attention", lambda q, k, v, sc, w=None, s=None: att(q, k, v, sc, w, None if s is None else s * sc)),
            "no_rotation": ("rotate_halves", lambda x, pos, r: x), "interleaved": ("rotate_halves", interleaved),
            "late_positions": ("rotate_halves", lambda x, pos, r: rot(x, pos if x.shape[1] == 2 else pos + 1, r)),
            "no_temperature": ("query_temperature", lambda pos, c: torch.ones(pos.shape, dtype=torch.float64)),
            "late_temperature": ("query_temperature", lambda pos, c: temp(pos - 1, c)),
            "unused_temperature": ("tempered_attention", own_keys),
            "late_read": ("selective_scan", late_read),
            "no_skip": ("selective_scan", lambda x, dt, A, B, C, D: scan(x, dt, A, B, C, D * 0)),
            "swapped_maps": ("selective_scan", lambda x, dt, A, B, C, D: scan(x, dt, A, C, B, D)),
            "no_step_in_input": ("selective_scan", lambda x, dt, A, B, C, D: scan(x / dt, dt, A, B, C, D * dt.mean())),
            "shifted_conv": ("short_conv", lambda x, w: conv(torch.cat([torch.zeros_like(x[:1]), x[:-1]]), w)),
            "linear_steps": ("softplus", lambda z: torch.clamp(z, min=0)),
            "one_best": ("choose_by_sigmoid", one_best),
            "no_groups": ("choose_by_sigmoid", lambda z, r: choose(z, {**r, "groups": None})),
            "no_router_scale": ("choose_by_sigmoid", lambda z, r: choose(z, {**r, "scale": 1.0})),
            "plain_weights": ("choose_by_sigmoid", lambda z, r: [(e, torch.sigmoid(z[e]) * r["scale"]) for e, _ in choose(z, r)]),
            "norm_without_one": ("rms_norm_around_zero", lambda x, w, e: norm(x, w - 1, e)),
            "no_cap": ("soft_cap", lambda x, c: x)}


@pytest.mark.parametrize("slip", sorted(_scan_slips()))
def test_a_mistake_in_a_scan_or_window_mechanism_shows(slip, monkeypatch):
    """Far above what 32-bit comparisons allow (5e-5) on many rows, and on some above the bf16 tolerance as well."""
    cfg = json.loads(json.dumps(hu.CONFIGS["scan_ragged"]))
    cfg["layers"][1]["mlp"] = hu.sigmoid_moe(12, 2, 20, 3, 1, 1.7, 28)
    w, toks = hu.weights(cfg, 5), hu.tokens(cfg, 48)
    right = oracle.forward(cfg, w, toks)
    fn, wrong = _scan_slips()[slip]
    monkeypatch.setattr(oracle, fn, wrong)
    e = hu.row_errors(oracle.forward(cfg, w, toks), right)
    assert float(e.max()) > 0.06 and float((e > 1e-3).double().mean()) > 0.25, (float(e.max()), float(e.median()))


def _side_slips():
    """Mistakes in Zigivik's mechanisms: name -> (function of the oracle, wrong version)."""
    att, halves, pairs, freq, conv, poly, low, norm, lat, kv, ff = (
        oracle.banded_attention, oracle.turn_halves, oracle.turn_pairs, oracle.yarn_frequencies, oracle.input_conv, oracle.poly_norm,
        oracle.low_rank_queries, oracle.one_number_norm, oracle.window_latent_attention, oracle.key_value_attention, oracle.poly_ff)

    def as_pairs(x, pos, r):
        n = r["dims"]
        order = torch.tensor([i // 2 + (i % 2) * (n // 2) for i in range(n)])
        out = x.clone()
        out[..., order] = halves(x[..., order], pos, r)
        return halves(x[..., torch.tensor([2 * i for i in range(n // 2)] + [2 * i + 1 for i in range(n // 2)])], pos, r)

    def as_halves(x, pos, r):
        n = r["dims"]
        order = torch.tensor([i // 2 + (i % 2) * (n // 2) for i in range(n)])
        out = x.clone()
        out[..., order] = pairs(x[..., order], pos, r)
        return out

    def own_values(h, W, p, c):                            # values behind the rotation
        T, G = h.shape[0], c["kv_heads"]
        pos = torch.arange(T)
        q = pairs((h @ W[p + "q"].T + W[p + "q.b"]).view(T, c["heads"], c["dim"]), pos, c["rot"])
        k = pairs((h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, c["dim"]), pos, c["rot"])
        return att(q, k, k, c["scale"], plus_one=True).reshape(T, -1) @ W[p + "o"].T

    def one_rms(z, act, eps):                              # every power divided by the rms of z itself
        n = oracle.rms(z, eps)
        return act[0] * n + act[1] * n ** 2 + act[2] * n ** 3 + act[3]

    def shifted(h, w):
        return h + conv(torch.cat([torch.zeros_like(h[:1]), h[:-1]]), w) - torch.cat([torch.zeros_like(h[:1]), h[:-1]])

    return {"window_longer": ("banded_attention", lambda q, k, v, s, w=None, plus_one=False: att(q, k, v, s, w and w + 1, plus_one)),
            "window_shorter": ("banded_attention", lambda q, k, v, s, w=None, plus_one=False: att(q, k, v, s, w and w - 1, plus_one)),
            "no_one": ("banded_attention", lambda q, k, v, s, w=None, plus_one=False: att(q, k, v, s, w)),
            "one_everywhere": ("banded_attention", lambda q, k, v, s, w=None, plus_one=False: att(q, k, v, s, w, True)),
            "as_pairs": ("turn_halves", as_pairs), "as_halves": ("turn_pairs", as_halves),
            "no_ramp": ("yarn_frequencies", lambda r: ([float(r["base"]) ** (-2.0 * i / r["dims"]) for i in range(r["dims"] // 2)], freq(r)[1])),
            "no_amplitude": ("yarn_frequencies", lambda r: (freq(r)[0], 1.0)),
            "amplitude_in_scale": ("yarn_frequencies", lambda r: (freq(r)[0], freq(r)[1] ** 2)),
            "late_positions": ("turn_pairs", lambda x, pos, r: pairs(x, pos if x.shape[1] == 2 else pos + 1, r)),
            "values_behind_rotation": ("key_value_attention", own_values),
            "no_conv": ("input_conv", lambda h, w: h), "conv_alone": ("input_conv", lambda h, w: conv(h, w) - h),
            "reversed_taps": ("input_conv", lambda h, w: conv(h, w.flip(1))), "shifted_conv": ("input_conv", shifted),
            "one_rms": ("poly_norm", one_rms), "no_constant": ("poly_norm", lambda z, a, e: poly(z, a, e) - a[3]),
            "swapped_powers": ("poly_norm", lambda z, a, e: poly(z, a[torch.tensor([2, 1, 0, 3])], e)),
            "no_query_norm": ("low_rank_queries", lambda h, W, p, e: (h @ W[p + "dq"].T) @ W[p + "uq"].T),
            "no_down_bias": ("poly_ff", lambda h, W, p, e: ff(h, W, p, e) - W[p + "down.b"]),
            "norm_around_zero": ("one_number_norm", lambda x, g, e: norm(x, 1 + g, e)),
            "own_latents": ("window_latent_attention", lambda h, W, p, c, e, kept: lat(h, W, p, c, e, {k: (a.flip(0), b) for k, (a, b) in kept.items()}
                                                                                       if c.get("kv_from") is not None else kept))}


@pytest.mark.parametrize("slip", sorted(_side_slips()))
def test_a_mistake_in_a_parallel_layer_shows(slip, monkeypatch):
    """Far above what 32-bit comparisons allow (5e-5) on many rows, and on some above the bf16 tolerance as well."""
    cfg = hu.CONFIGS["side_ragged"]
    w, toks = hu.weights(cfg, 5), hu.tokens(cfg, 60)
    right = oracle.forward(cfg, w, toks)
    fn, wrong = _side_slips()[slip]
    monkeypatch.setattr(oracle, fn, wrong)
    e = hu.row_errors(oracle.forward(cfg, w, toks), right)
    assert float(e.max()) > 0.06 and float((e > 1e-3).double().mean()) > 0.25, (float(e.max()), float(e.median()))

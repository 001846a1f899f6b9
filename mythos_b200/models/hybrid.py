"""Weights of a layer-list model (:mod:`.hybrid_config`) under their checkpoint names.

The model object holds tensors; the computation is the inference engine's
(:mod:`mythos_b200.infer.hybrid`), which packs them into the layouts its kernels read. ``forward`` runs
whole sequences through such an engine, so the model-level helpers (log-probabilities, beam search,
embeddings, reranking) work as they do for the other models. There is no CPU forward.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .hybrid_config import (AttentionMixer, HybridConfig, LatentAttentionMixer, MoeFF, ParallelMixer,
                            RecurrentMixer, SelectiveMixer)


def _attention_shapes(p: str, m: AttentionMixer, d: int) -> dict:
    out = {p + "q": (m.heads * m.dim, d)}
    if m.kv_from is None:
        out[p + "k"] = (m.kv_heads * m.dim, d)
        if m.values == "own":
            out[p + "v"] = (m.kv_heads * m.vdim, d)
    if m.bias:
        out.update({name + ".b": shape[:1] for name, shape in out.items()})
    if m.qk_norm == "weighted":
        out[p + "q.norm"] = (m.dim,)
        if m.kv_from is None:
            out[p + "k.norm"] = (m.dim,)
    if m.gate is not None:
        out[p + "g"] = (m.heads * (m.vdim if m.gate == "channel" else 1), d)
    if m.sink == "learned":
        out[p + "sink"] = (m.heads,)
    out[p + "o"] = (d, m.heads * m.vdim)
    return out


def _selective_shapes(p: str, m: SelectiveMixer, d: int) -> dict:
    c = m.inner
    return {p + "in": (2 * c, d), p + "conv": (c, m.conv), p + "conv.b": (c,), p + "x": (m.dt_rank + 2 * m.state, c),
            p + "dt": (c, m.dt_rank), p + "dt.b": (c,), p + "A_log": (c, m.state), p + "D": (c,), p + "o": (d, c)}


def _gla_shapes(p: str, m: RecurrentMixer, d: int) -> dict:
    return {p + "q": (m.heads * m.dim, d), p + "k": (m.heads * m.dim, d), p + "v": (m.heads * m.vdim, d),
            p + "g": (m.heads * m.vdim, d), p + "o": (d, m.heads * m.vdim), p + "norm": (m.vdim,),
            p + "a1": (None, d), p + "a2": (m.heads * m.dim, None), p + "a2.b": (m.heads * m.dim,)}


def _delta_shapes(p: str, m: RecurrentMixer, d: int) -> dict:
    cq, cv = m.kv_heads * m.dim, m.heads * m.vdim
    out = {p + "q": (cq, d), p + "k": (cq, d), p + "v": (cv, d), p + "b": (m.heads, d), p + "A_log": (m.heads,),
           p + "norm": (m.vdim,), p + "a1": (None, d), p + "a2": (m.heads * m.dim, None),
           p + "dt_bias": (m.heads * m.dim,), p + "g1": (None, d), p + "g2": (cv, None), p + "o": (d, cv)}
    out.update({p + "q.conv": (cq, m.conv), p + "k.conv": (cq, m.conv), p + "v.conv": (cv, m.conv)})
    return out


def _latent_shapes(p: str, m: LatentAttentionMixer, d: int) -> dict:
    q = m.heads * (m.dim + m.rot_dim)
    out = {p + "dq": (m.q_rank, d), p + "dq.norm": (m.q_rank,), p + "uq": (q, m.q_rank)} if m.q_rank else {p + "q": (q, d)}
    if m.kv_from is None:
        out.update({p + "dkv": (m.kv_rank + m.rot_dim, d), p + "dkv.norm": (m.kv_rank,)})
    out.update({p + "uk": (m.heads * m.dim, m.kv_rank), p + "uv": (m.heads * m.vdim, m.kv_rank)})
    if m.sink == "learned":
        out[p + "sink"] = (m.heads,)
    if m.gate:
        out[p + "g"] = (m.heads * m.vdim, d)
    out[p + "o"] = (d, m.heads * m.vdim)
    return out


def _gated_shapes(p: str, ff: int, d: int) -> dict:
    return {p + "gate": (ff, d), p + "up": (ff, d), p + "down": (d, ff)}


def _mlp_shapes(p: str, f, d: int) -> dict:
    if not isinstance(f, MoeFF):
        if f.gated:
            return _gated_shapes(p, f.ff, d)
        return {p + "up": (f.ff, d), p + "up.b": (f.ff,), p + "down": (d, f.ff), p + "down.b": (d,), p + "act": (4,)}
    out = {p + "router": (f.experts, d)}
    if f.correction:
        out[p + "correction"] = (f.experts,)
    if f.shared:
        out.update(_gated_shapes(p + "shared.", f.shared, d))
    for e in range(f.experts):
        out.update(_gated_shapes(p + f"e{e}.", f.ff, d))
    return out


def expected_shapes(cfg: HybridConfig) -> dict:
    """Name -> shape of every tensor; ``None`` marks a low-rank width that the tensors themselves fix."""
    d = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, d)}
    if cfg.position_table:
        out["pos"] = (cfg.max_seq_len, d)
    norm = () if cfg.scalar_norms else (d,)
    out["final.norm"] = norm
    if cfg.embed_norm:
        out["embed.norm"] = norm
    if not cfg.tied_head:
        out["head"] = (cfg.vocab_size, d)
    if cfg.token_side:
        out["side.embed"] = (cfg.vocab_size, cfg.num_layers * cfg.token_side)

    def norms(p: str, n: int) -> None:                 # a sublayer's norms: before (if the design has one), after
        out[p + f"norm{n}"] = norm
        if cfg.pre_norm and cfg.post_norm:
            out[p + f"norm{n}b"] = norm

    for i, spec in enumerate(cfg.layers):
        p = f"l{i}."
        norms(p, 1)
        if cfg.input_conv:
            out[p + "canon1"] = (d, cfg.input_conv)
        m = spec.mixer
        if isinstance(m, ParallelMixer):
            right = _selective_shapes if isinstance(m.right, SelectiveMixer) else _delta_shapes
            out.update(_attention_shapes(p + "mix.left.", m.left, d))
            out.update(right(p + "mix.right.", m.right, d))
            if m.scales is None:
                out[p + "mix.left.out"] = out[p + "mix.right.out"] = (d,)
        elif isinstance(m, AttentionMixer):
            out.update(_attention_shapes(p + "mix.", m, d))
        elif isinstance(m, LatentAttentionMixer):
            out.update(_latent_shapes(p + "mix.", m, d))
        else:
            out.update(_gla_shapes(p + "mix.", m, d))
        if spec.mlp is not None:
            if not cfg.parallel:
                norms(p, 2)
            out.update(_mlp_shapes(p + "mlp.", spec.mlp, d))
        if cfg.token_side:
            out.update({p + "side.gate": (cfg.token_side, d), p + "side.proj": (d, cfg.token_side), p + "side.norm": (d,)})
    return out


def _key(name: str) -> str:
    return name.replace(".", "/")


class HybridModel(nn.Module):
    def __init__(self, cfg: HybridConfig, tensors: dict):
        super().__init__()
        self.cfg = cfg
        self._engine = None
        for name, shape in expected_shapes(cfg).items():
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            t = tensors[name]
            if t.dim() != len(shape) or any(w is not None and int(w) != n for w, n in zip(shape, t.shape)):
                raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the configuration wants {shape}")
            self.register_parameter(_key(name), nn.Parameter(t, requires_grad=False))

    def tensor(self, name: str) -> torch.Tensor:
        return getattr(self, _key(name)).detach()

    def named_tensors(self):
        return [(n.replace("/", "."), p.detach()) for n, p in self.named_parameters()]

    @classmethod
    def random(cls, cfg: HybridConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16, low_rank: int = 16,
               std: float = 0.02) -> "HybridModel":
        """Random weights of this configuration (benchmarks, tests)."""
        g = torch.Generator(device=device).manual_seed(seed)
        out = {}
        for name, shape in expected_shapes(cfg).items():
            shape = tuple(low_rank if n is None else n for n in shape)
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("norm", "norm1", "norm2", "norm1b", "norm2b", "out"):
                t = torch.full(shape, 1.0 - cfg.norm_offset, device=device)
            elif leaf == "A_log" and len(shape) == 2:
                t = torch.log(torch.arange(1, shape[1] + 1, device=device, dtype=torch.float32)).expand(shape)
            elif leaf == "act":
                t = torch.tensor([0.6, 0.3, 0.2, 0.0], device=device)
            elif leaf == "D":
                t = torch.ones(shape, device=device)
            elif name.endswith(".dt.b"):
                t = -5.0 + 3.0 * torch.rand(shape, device=device, generator=g)
            elif name.endswith((".q.b", ".k.b", ".v.b", ".conv.b", ".up.b", ".down.b")):
                t = torch.randn(shape, device=device, generator=g) * std
            elif leaf == "A_log":
                t = torch.log(1.0 + 3.0 * torch.rand(shape, device=device, generator=g))
            elif leaf in ("sink", "correction"):
                t = torch.randn(shape, device=device, generator=g) * (1.0 if leaf == "sink" else 0.01)
            elif leaf == "dt_bias":
                t = -4.0 + torch.rand(shape, device=device, generator=g)
            elif leaf == "b":
                t = (torch.rand(shape, device=device, generator=g) * 4 + 1 if len(shape) == 1
                     else torch.randn(shape, device=device, generator=g) * std)
            else:
                t = torch.randn(shape, device=device, generator=g) * ({"conv": 0.5, "canon1": 0.25}.get(leaf, std))
            out[name] = t.to(dtype)
        return cls(cfg, out)

    def param_count(self) -> int:
        return sum(p.numel() for p in self.parameters())

    # ------------------------------------------------------------------ whole-sequence forward
    def engine(self):
        """Engine behind :meth:`forward` (built on first use, one sequence at a time)."""
        dev = self.tensor("embed").device
        if dev.type != "cuda":
            raise RuntimeError("a layer-list model runs on the GPU only; move it to a CUDA device")
        if self._engine is None:
            from ..infer.engine import InferenceEngine

            self._engine = InferenceEngine.from_model(self, device=dev, max_batch=1, max_seq_len=self.cfg.max_seq_len)
        return self._engine

    def _rows(self, ids, fn):
        eng = self.engine()
        out = []
        for row in torch.as_tensor(ids).tolist():
            seq = eng.cache.new_sequence()
            try:
                out.append(fn(eng, seq, row))
            finally:
                eng.release(seq)
        return torch.stack(out)

    def hidden_states(self, ids, pos=None):
        """ids int [B, S] -> final normalised hidden states [B, S, d]."""
        return self._rows(ids, lambda e, s, row: e.step_hidden([s], [row])[0][:, : self.cfg.hidden_size])

    def forward(self, ids, targets=None, pos=None):
        """Logits [B, S, V] (fp32)."""
        if targets is not None:
            raise NotImplementedError("layer-list models are inference only")
        return self._rows(ids, lambda e, s, row: e.step([s], [row], [list(range(len(row)))]))

    def logits(self, h):
        return self.engine()._logits(h.reshape(-1, h.shape[-1])).view(*h.shape[:-1], -1)

"""Configuration of layer-list ("hybrid") designs: every layer names its mixer and its feed-forward.

Mixers (``LayerSpec.mixer``):

* ``RecurrentMixer`` kind ``gla``: gated linear attention, decay ``sigmoid(z)^(1/tau)`` per key channel;
* ``RecurrentMixer`` kind ``delta``: gated delta rule with short convolutions and unit-norm q / k;
* ``AttentionMixer``: causal softmax attention without rotation, q / k norms, per-head output gate,
  key and value widths of their own;
* ``ParallelMixer``: an attention and a delta mixer on the same input, averaged after their own norms;
* ``LatentAttentionMixer``: attention whose keys and values are linear maps of one normalised latent per
  token, plus a rotated key part that all heads share; only the latent and that part are cached. A
  learned sink per head enters the softmax denominator.

Feed-forwards (``LayerSpec.mlp``): ``DenseFF`` (gated, with its activation) and ``MoeFF`` (softmax router
with a choice correction and expert groups over gated experts).

The designs served under this configuration are Teganex (norms before and after every sublayer, learned
positions) and Lebedra (norms on the sublayer outputs only, latent attention, experts, per-layer token input).
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .registry import register


@dataclass
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float

    def __post_init__(self):
        _positive(self, "heads", "kv_heads", "dim", "vdim")
        if self.heads % self.kv_heads:
            raise ValueError(f"attention: {self.heads} heads do not divide by {self.kv_heads} key/value heads")


@dataclass
class RecurrentMixer:
    kind: str                  # "gla" | "delta"
    heads: int
    kv_heads: int              # heads of q and k (gla: = heads)
    dim: int
    vdim: int
    tau: float = 1.0           # gla: decay = sigmoid(z)^(1/tau)
    conv: int = 0              # taps of the short convolution on q, k, v (0: none)

    def __post_init__(self):
        _positive(self, "heads", "kv_heads", "dim", "vdim")
        if self.kind not in ("gla", "delta"):
            raise ValueError(f"recurrent mixer: unknown kind {self.kind!r}")
        if self.heads % self.kv_heads:
            raise ValueError(f"recurrent mixer: {self.heads} heads do not divide by {self.kv_heads} q/k heads")

    @property
    def conv_channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass
class ParallelMixer:
    left: AttentionMixer
    right: RecurrentMixer


@dataclass
class LatentAttentionMixer:
    heads: int
    dim: int                   # unrotated query / key width of a head
    rot_dim: int               # rotated query / key width (the key part is shared by all heads)
    vdim: int
    kv_rank: int               # width of the latent
    scale: float
    rot_base: float

    def __post_init__(self):
        _positive(self, "heads", "dim", "rot_dim", "vdim", "kv_rank")
        if self.rot_dim % 2:
            raise ValueError(f"latent attention: the rotated width must be even, got {self.rot_dim}")


@dataclass
class DenseFF:
    """``down(act(gate h) * (up h))``"""
    ff: int
    act: str = "silu"          # "silu" | "relu"

    def __post_init__(self):
        _positive(self, "ff")
        if self.act not in ("silu", "relu"):
            raise ValueError(f"feed-forward: unknown activation {self.act!r}")


@dataclass
class MoeFF:
    """``top`` of ``experts`` clamped gated experts of width ``ff``: g = min(gate h, limit),
    u = clamp(up h, -limit, limit), ``down(g sigmoid(alpha g) (u + 1))``. Scores are the softmax over all
    experts and weigh the outputs as they are; scores + correction choose, first the ``keep`` best of
    ``groups`` groups of neighbours (by their best expert), then the experts in them."""
    experts: int
    top: int
    ff: int
    limit: float
    groups: int = 1
    keep: int = 1
    alpha: float = 1.702

    def __post_init__(self):
        _positive(self, "experts", "top", "ff", "groups", "keep")
        if self.experts % self.groups or self.keep > self.groups:
            raise ValueError(f"experts: {self.experts} do not form {self.groups} equal groups, or more are kept ({self.keep})")
        if self.top > self.experts // self.groups * self.keep:
            raise ValueError(f"experts: {self.top} of {self.experts // self.groups * self.keep} eligible ones")


@dataclass
class LayerSpec:
    type: str
    mixer: object
    mlp: DenseFF | MoeFF | None = None

    @property
    def attention(self) -> AttentionMixer | None:
        return self.mixer.left if isinstance(self.mixer, ParallelMixer) else None

    @property
    def latent(self) -> LatentAttentionMixer | None:
        return self.mixer if isinstance(self.mixer, LatentAttentionMixer) else None

    @property
    def recurrent(self) -> RecurrentMixer | None:
        if isinstance(self.mixer, ParallelMixer):
            return self.mixer.right
        return self.mixer if isinstance(self.mixer, RecurrentMixer) else None


DEFAULT_CONTEXT = 8192        # of designs without a position table, where the caller names no length
LONGEST_CONTEXT = 1 << 20     # positions the engine accepts for them


@dataclass
class HybridConfig:
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    max_seq_len: int = DEFAULT_CONTEXT
    architecture: str = "Teganex"
    position_table: bool = True    # learned positions, ``max_seq_len`` rows
    pre_norm: bool = True          # sublayers read a normalised copy of the stream (else the stream itself)
    residual_mult: float = 1.0     # x <- x + residual_mult * norm(sublayer)
    token_side: int = 0            # width of the per-layer token input, 0: none
    extras: dict = field(default_factory=dict)

    def __post_init__(self):
        _positive(self, "vocab_size", "hidden_size", "max_seq_len")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def context_limit(self) -> int:
        return self.max_seq_len if self.position_table else LONGEST_CONTEXT

    # ------------------------------------------------------------------ config.json
    @classmethod
    def from_dict(cls, d: dict) -> "HybridConfig":
        arch = str(d["architecture"])
        common = dict(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float(d["norm"]["eps"]), architecture=arch)
        if arch == "Lebedra":
            side = d.get("token_side")
            return cls(layers=[_layer_from_dict(i, x, ("latent_attention",), "relu") for i, x in enumerate(d["layers"])],
                       position_table=False, pre_norm=False, residual_mult=float(d["residual_mult"]),
                       token_side=int(side["dim"]) if side else 0, **common)
        return cls(layers=[_layer_from_dict(i, x, ("gla", "parallel"), "silu") for i, x in enumerate(d["layers"])],
                   embed_scale=float(d["embedding"]["scale"]), logit_scale=float(d["logit_scale"]),
                   max_seq_len=int(d["max_positions"]), **common)

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "layers": [_layer_to_dict(x) for x in self.layers]}
        if self.architecture == "Lebedra":
            d["residual_mult"] = self.residual_mult
            if self.token_side:
                d["token_side"] = {"dim": self.token_side}
        else:
            d.update(max_positions=self.max_seq_len, embedding={"scale": self.embed_scale}, logit_scale=self.logit_scale)
        return d


def _positive(obj, *names):
    for n in names:
        if int(getattr(obj, n)) <= 0:
            raise ValueError(f"{type(obj).__name__}.{n} must be positive, got {getattr(obj, n)!r}")


def _layer_from_dict(index: int, d: dict, kinds: tuple, act: str) -> LayerSpec:
    kind, m = d["type"], d["mixer"]
    if kind not in kinds:
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    if kind == "gla":
        mixer = RecurrentMixer("gla", int(m["heads"]), int(m["heads"]), int(m["dim"]), int(m["vdim"]), tau=float(m["tau"]))
    elif kind == "parallel":
        a, r = m["left"], m["right"]
        mixer = ParallelMixer(
            AttentionMixer(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"])),
            RecurrentMixer("delta", int(r["heads"]), int(r["kv_heads"]), int(r["dim"]), int(r["vdim"]), conv=int(r["conv"])))
    else:
        rot = m["rot"]
        if int(rot.get("dims", m["rot_dim"])) != int(m["rot_dim"]):
            raise ValueError(f"layer {index}: rotated dimensions {rot['dims']} and rotated width {m['rot_dim']} differ")
        mixer = LatentAttentionMixer(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                     float(m["scale"]), float(rot["base"]))
    return LayerSpec(kind, mixer, _mlp_from_dict(index, d.get("mlp"), act))


def _mlp_from_dict(index: int, mlp: dict | None, act: str) -> DenseFF | MoeFF | None:
    if mlp is None:
        return None
    if mlp.get("kind") == "dense":
        return DenseFF(int(mlp["ff"]), act)
    if mlp.get("kind") == "moe" and act == "relu":
        e, r = mlp["expert"], mlp["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        return MoeFF(int(r["experts"]), int(r["top"]), int(e["ff"]), float(e["limit"]), int(g["count"]), int(g["keep"]))
    raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")


def _layer_to_dict(x: LayerSpec) -> dict:
    m = x.mixer
    if isinstance(m, ParallelMixer):
        mixer = {"left": {"heads": m.left.heads, "kv_heads": m.left.kv_heads, "dim": m.left.dim, "vdim": m.left.vdim,
                          "scale": m.left.scale},
                 "right": {"heads": m.right.heads, "kv_heads": m.right.kv_heads, "dim": m.right.dim, "vdim": m.right.vdim,
                           "conv": m.right.conv}}
    elif isinstance(m, LatentAttentionMixer):
        mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale,
                 "rot": {"base": m.rot_base, "dims": m.rot_dim}}
    else:
        mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}
    f = x.mlp
    if isinstance(f, MoeFF):
        mlp = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit},
               "router": {"experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}
    else:
        mlp = {"kind": "dense", "ff": f.ff} if f is not None else None
    return {"type": x.type, "mixer": mixer, "mlp": mlp}


# ------------------------------------------------------------------ named configurations
def teganex_config(width: int = 2048, layers: int = 8, vocab: int = 32000, max_positions: int = 8192,
                   parallel_every: int = 4) -> HybridConfig:
    """Teganex at the layer sizes of a 1-2B model: every ``parallel_every``-th layer is a parallel layer
    (16 query heads over 2 key heads, 128-wide; 16 delta heads), the others gated linear attention."""
    h = width // 128
    out = []
    for i in range(layers):
        if i % parallel_every == parallel_every - 1:
            out.append(LayerSpec("parallel", ParallelMixer(
                AttentionMixer(h, max(1, h // 8), 128, 128, 128 ** -0.5),
                RecurrentMixer("delta", h, h, 128, 128, conv=4)), DenseFF(width * 11 // 4 // 128 * 128)))
        else:
            out.append(LayerSpec("gla", RecurrentMixer("gla", h, h, 64, 128, tau=16.0), DenseFF(width * 11 // 4 // 128 * 128)))
    return HybridConfig(vocab, width, out, 1e-6, 1.0, 1.0, max_positions)


def lebedra_config(width: int = 2048, layers: int = 8, vocab: int = 32000, max_positions: int = 8192, experts: int = 64,
                   top: int = 6) -> HybridConfig:
    """Lebedra at the layer sizes of a real model: latents of 512 with heads of 128 + 64 rotated, a dense first
    layer, then experts whose ``top`` together are about as wide as the dense feed-forward."""
    mixer = LatentAttentionMixer(width // 128, 128, 64, 128, 512, 192 ** -0.5, 10000.0)
    dense = width * 11 // 4 // 128 * 128
    moe = MoeFF(experts, top, max(128, dense // top // 128 * 128), 7.0, 8, 3)
    out = [LayerSpec("latent_attention", mixer, DenseFF(dense, "relu") if i == 0 else moe) for i in range(layers)]
    return HybridConfig(vocab, width, out, 1e-6, max_seq_len=max_positions, architecture="Lebedra", position_table=False,
                        pre_norm=False, residual_mult=0.5, token_side=128)


register("Lebedra", HybridConfig.from_dict, "mythos_b200.models.hybrid:HybridModel")
register("Teganex", HybridConfig.from_dict, "mythos_b200.models.hybrid:HybridModel")

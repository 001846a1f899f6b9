"""Configuration of layer-list ("hybrid") designs: every layer names its mixer and its feed-forward.

Mixers (``LayerSpec.mixer``):

* ``RecurrentMixer`` kind ``gla``: gated linear attention, decay ``sigmoid(z)^(1/tau)`` per key channel;
* ``RecurrentMixer`` kind ``delta``: gated delta rule with short convolutions and unit-norm q / k;
* ``AttentionMixer``: causal softmax attention without rotation, q / k norms, per-head output gate,
  key and value widths of their own;
* ``ParallelMixer``: an attention and a delta mixer on the same input, averaged after their own norms.

The design served today under this configuration is Teganex.
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
class LayerSpec:
    type: str
    mixer: object
    ff: int = 0                # width of the gated feed-forward, 0: the layer has none

    @property
    def attention(self) -> AttentionMixer | None:
        return self.mixer.left if isinstance(self.mixer, ParallelMixer) else None

    @property
    def recurrent(self) -> RecurrentMixer | None:
        return self.mixer.right if isinstance(self.mixer, ParallelMixer) else self.mixer


@dataclass
class HybridConfig:
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    embed_scale: float
    logit_scale: float
    max_seq_len: int           # rows of the learned position table
    architecture: str = "Teganex"
    extras: dict = field(default_factory=dict)

    def __post_init__(self):
        _positive(self, "vocab_size", "hidden_size", "max_seq_len")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    # ------------------------------------------------------------------ config.json
    @classmethod
    def from_dict(cls, d: dict) -> "HybridConfig":
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                   layers=[_layer_from_dict(i, x) for i, x in enumerate(d["layers"])],
                   norm_eps=float(d["norm"]["eps"]), embed_scale=float(d["embedding"]["scale"]),
                   logit_scale=float(d["logit_scale"]), max_seq_len=int(d["max_positions"]),
                   architecture=str(d["architecture"]))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                "max_positions": self.max_seq_len, "embedding": {"scale": self.embed_scale},
                "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale,
                "layers": [_layer_to_dict(x) for x in self.layers]}


def _positive(obj, *names):
    for n in names:
        if int(getattr(obj, n)) <= 0:
            raise ValueError(f"{type(obj).__name__}.{n} must be positive, got {getattr(obj, n)!r}")


def _layer_from_dict(index: int, d: dict) -> LayerSpec:
    kind, m, mlp = d["type"], d["mixer"], d.get("mlp")
    if kind == "gla":
        mixer = RecurrentMixer("gla", int(m["heads"]), int(m["heads"]), int(m["dim"]), int(m["vdim"]), tau=float(m["tau"]))
    elif kind == "parallel":
        a, r = m["left"], m["right"]
        mixer = ParallelMixer(
            AttentionMixer(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"])),
            RecurrentMixer("delta", int(r["heads"]), int(r["kv_heads"]), int(r["dim"]), int(r["vdim"]), conv=int(r["conv"])))
    else:
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    ff = 0
    if mlp is not None:
        if mlp.get("kind") != "dense":
            raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")
        ff = int(mlp["ff"])
        if ff <= 0:
            raise ValueError(f"layer {index}: feed-forward width must be positive")
    return LayerSpec(kind, mixer, ff)


def _layer_to_dict(x: LayerSpec) -> dict:
    m = x.mixer
    if isinstance(m, ParallelMixer):
        mixer = {"left": {"heads": m.left.heads, "kv_heads": m.left.kv_heads, "dim": m.left.dim, "vdim": m.left.vdim,
                          "scale": m.left.scale},
                 "right": {"heads": m.right.heads, "kv_heads": m.right.kv_heads, "dim": m.right.dim, "vdim": m.right.vdim,
                           "conv": m.right.conv}}
    else:
        mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}
    return {"type": x.type, "mixer": mixer, "mlp": {"kind": "dense", "ff": x.ff} if x.ff else None}


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
                RecurrentMixer("delta", h, h, 128, 128, conv=4)), ff=width * 11 // 4 // 128 * 128))
        else:
            out.append(LayerSpec("gla", RecurrentMixer("gla", h, h, 64, 128, tau=16.0), ff=width * 11 // 4 // 128 * 128))
    return HybridConfig(vocab, width, out, 1e-6, 1.0, 1.0, max_positions)


register("Teganex", HybridConfig.from_dict, "mythos_b200.models.hybrid:HybridModel")

"""Configuration of layer-list ("hybrid") designs: every layer names its mixer and its feed-forward.

Mixers (``LayerSpec.mixer``):

* ``RecurrentMixer`` kind ``gla``: gated linear attention, decay ``sigmoid(z)^(1/tau)`` per key channel;
* ``RecurrentMixer`` kind ``delta``: gated delta rule with short convolutions and unit-norm q / k;
* ``AttentionMixer``: causal softmax attention with key and value widths of their own; q / k norms, biases,
  rotation, query temperature, sliding window, sink and output gate as its fields say. A layer may use the
  keys and values of an earlier one (``kv_from``);
* ``SelectiveMixer``: selective scan, a diagonal recurrence per channel with step sizes, input and output maps
  that depend on the token, behind a short convolution;
* ``ParallelMixer``: an attention and a recurrent mixer on the same input, averaged after their own norms or
  added with constant scales;
* ``LatentAttentionMixer``: attention whose keys and values are linear maps of one normalised latent per
  token, plus a rotated key part that all heads share; only the latent and that part are cached. Low-rank queries,
  sliding window, sink and output gate as its fields say; a layer may use an earlier one's latents (``kv_from``).

Feed-forwards (``LayerSpec.mlp``): ``DenseFF`` (gated, or one projection and a polynomial of normalised powers) and
``MoeFF`` (a router that scores by softmax or sigmoid, with expert groups, over gated experts, and optionally a shared
expert).

The designs served under this configuration are Teganex (norms before and after every sublayer, learned
positions), Lebedra (norms on the sublayer outputs only, latent attention, experts, per-layer token input),
Dogozen (norms around sublayers with weights stored around zero, tempered full attention with shared caches,
window attention beside a selective scan, sigmoid-routed experts, tied and soft-capped output) and Zigivik (mixer and
feed-forward side by side behind one norm with a single weight, a short convolution in front of every mixer, window
latent attention with shared latents, attention whose values are its keys).
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field

from .registry import register


@dataclass
class FrequencyScaling:
    """Slows the rotation of pairs that turn fewer than ``low`` times within ``original`` positions by ``factor``,
    leaves those that turn more than ``high`` times, and blends between."""
    factor: float
    low: float
    high: float
    original: float

    def apply(self, f: float) -> float:
        turns = self.original * f / (2.0 * math.pi)
        if turns > self.high:
            return f
        if turns < self.low:
            return f / self.factor
        s = (turns - self.low) / (self.high - self.low) if self.high != self.low else 1.0
        return (1.0 - s) * f / self.factor + s * f


@dataclass
class RampScaling:
    """YaRN: slows pairs by ``factor`` along a ramp over their number, from the pair that turns ``fast`` times within
    ``original`` positions (not slowed) to the one that turns ``slow`` times; what is rotated grows by ``amplitude``."""
    factor: float
    original: float
    fast: float
    slow: float

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    def ramp(self, base: float, dims: int) -> list:
        """Share of the slowed frequency in every pair's."""
        def pair(turns: float) -> float:
            return dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo, hi = max(math.floor(pair(self.fast)), 0), min(math.ceil(pair(self.slow)), dims - 1)
        return [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]


@dataclass
class Rotation:
    """Rotary positions on the first ``dims`` columns of a head: column i paired with i + dims / 2 (``halves``) or
    column 2i with 2i + 1 (``pairs``)."""
    base: float
    dims: int
    scaling: FrequencyScaling | RampScaling | None = None
    layout: str = "halves"

    def turns(self) -> list:
        """Revolutions per position of every pair."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if isinstance(self.scaling, RampScaling):
            f = [x / self.scaling.factor * r + x * (1.0 - r) for x, r in zip(f, self.scaling.ramp(self.base, self.dims))]
        elif self.scaling:
            f = [self.scaling.apply(x) for x in f]
        return [x / (2.0 * math.pi) for x in f]

    @property
    def amplitude(self) -> float:
        """Factor of cosines and sines."""
        return self.scaling.amplitude if isinstance(self.scaling, RampScaling) else 1.0


@dataclass
class QueryTemperature:
    """Queries at position p are multiplied by 1 + coef ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: float


SINKS = ("learned", "zero", None)


@dataclass
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    qk_norm: str | None = "weighted"   # RMS norm of every q / k head: "weighted", "plain" (no weight) or None
    gate: str | None = "head"          # sigmoid output gate: one value per head, per "channel", or None
    bias: bool = False                 # on q, k and v
    values: str = "own"                # "own", or "keys": the projected keys, before norm and rotation
    rotation: Rotation | None = None
    window: int = 0                    # keys a query sees, itself included; 0: all earlier ones
    sink: str | None = None            # one more logit per head in the softmax denominator: "learned", or "zero"
    q_temp: QueryTemperature | None = None
    kv_from: int | None = None         # layer whose cached keys and values are used

    def __post_init__(self):
        _positive(self, "heads", "kv_heads", "dim", "vdim")
        if self.heads % self.kv_heads:
            raise ValueError(f"attention: {self.heads} heads do not divide by {self.kv_heads} key/value heads")
        if self.qk_norm not in ("weighted", "plain", None) or self.gate not in ("head", "channel", None):
            raise ValueError(f"attention: unknown norm {self.qk_norm!r} or gate {self.gate!r}")
        if self.window < 0:
            raise ValueError(f"attention: negative window {self.window}")
        if self.sink not in SINKS or self.values not in ("own", "keys"):
            raise ValueError(f"attention: unknown sink {self.sink!r} or values {self.values!r}")
        if self.values == "keys" and self.dim != self.vdim:
            raise ValueError(f"attention: keys of width {self.dim} cannot be values of width {self.vdim}")
        r = self.rotation
        if r is not None and (r.dims <= 0 or r.dims % 2 or r.dims > self.dim):
            raise ValueError(f"attention: {r.dims} rotated columns of {self.dim}")
        if self.q_temp is not None and self.q_temp.every <= 0:
            raise ValueError("attention: the query temperature's period must be positive")


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
class SelectiveMixer:
    """S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n, y_c = sum_n S[c, n] C_n + D_c x_c, times silu(z)."""
    inner: int                 # channels
    state: int                 # state values per channel
    dt_rank: int               # width of the low-rank map to the step sizes
    conv: int                  # taps of the short convolution on x

    def __post_init__(self):
        _positive(self, "inner", "state", "dt_rank", "conv")


@dataclass
class ParallelMixer:
    left: AttentionMixer
    right: RecurrentMixer | SelectiveMixer
    scales: tuple | None = None        # (left, right) factors of the sum; None: mean of the normalised outputs


@dataclass
class LatentAttentionMixer:
    heads: int
    dim: int                   # unrotated query / key width of a head
    rot_dim: int               # rotated query / key width (the key part is shared by all heads)
    vdim: int
    kv_rank: int               # width of the latent
    scale: float
    rotation: Rotation         # of all rot_dim columns
    q_rank: int = 0            # queries are a map of a normalised vector of this width, 0: of the input itself
    window: int = 0            # keys a query sees, itself included; 0: all earlier ones
    sink: str | None = "learned"
    gate: bool = False         # sigmoid output gate per channel
    kv_from: int | None = None # layer whose cached latents and rotated key parts are used

    def __post_init__(self):
        _positive(self, "heads", "dim", "rot_dim", "vdim", "kv_rank")
        if self.rot_dim % 2:
            raise ValueError(f"latent attention: the rotated width must be even, got {self.rot_dim}")
        if self.rotation.dims != self.rot_dim:
            raise ValueError(f"latent attention: rotated dimensions {self.rotation.dims} and rotated width {self.rot_dim} differ")
        if self.sink not in SINKS or self.window < 0 or self.q_rank < 0:
            raise ValueError(f"latent attention: sink {self.sink!r}, window {self.window} or query rank {self.q_rank}")


@dataclass
class DenseFF:
    """``down(act(gate h) * (up h))``; with ``act`` "poly_norm" ``down(act(up h + b)) + b``, where act(z) is
    a N(z) + b N(z^2) + c N(z^3) + e of four weights, N dividing a token's vector by its root mean square."""
    ff: int
    act: str = "silu"          # "silu" | "relu" | "poly_norm"

    def __post_init__(self):
        _positive(self, "ff")
        if self.act not in ("silu", "relu", "poly_norm"):
            raise ValueError(f"feed-forward: unknown activation {self.act!r}")

    @property
    def gated(self) -> bool:
        return self.act != "poly_norm"


@dataclass
class MoeFF:
    """``top`` of ``experts`` gated experts of width ``ff``. Scores (softmax over all experts, or the sigmoid of each)
    choose, plus a correction per expert if there is one: first the ``keep`` best of ``groups`` groups of neighbours
    (by the sum of their ``group_best`` largest), then the experts in them. The chosen scores, without
    correction, weigh the outputs: as they are, or normalised to the sum ``scale``. A shared expert of width
    ``shared`` runs for every token.

    Experts: ``act`` "clamped": g = min(gate h, limit), u = clamp(up h, -limit, limit),
    ``down(g sigmoid(alpha g) (u + 1))``; "silu" / "relu": as ``DenseFF``."""
    experts: int
    top: int
    ff: int
    limit: float = 0.0
    groups: int = 1
    keep: int = 1
    alpha: float = 1.702
    act: str = "clamped"
    score: str = "softmax"     # "softmax" | "sigmoid"
    correction: bool = True
    group_best: int = 1        # scores of a group that are added (1 or 2)
    normalise: bool = False
    scale: float = 1.0
    shared: int = 0

    def __post_init__(self):
        _positive(self, "experts", "top", "ff", "groups", "keep")
        if self.act not in ("clamped", "silu", "relu") or self.score not in ("softmax", "sigmoid") or self.group_best not in (1, 2):
            raise ValueError(f"experts: unknown activation {self.act!r}, score {self.score!r} or group rule {self.group_best!r}")
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
        m = self.mixer.left if isinstance(self.mixer, ParallelMixer) else self.mixer
        return m if isinstance(m, AttentionMixer) else None

    @property
    def latent(self) -> LatentAttentionMixer | None:
        return self.mixer if isinstance(self.mixer, LatentAttentionMixer) else None

    @property
    def recurrent(self) -> RecurrentMixer | SelectiveMixer | None:
        m = self.mixer.right if isinstance(self.mixer, ParallelMixer) else self.mixer
        return m if isinstance(m, (RecurrentMixer, SelectiveMixer)) else None


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
    post_norm: bool = True         # sublayer outputs are normalised before they are added
    parallel: bool = False         # mixer and feed-forward read the same norm and are added together
    scalar_norms: bool = False     # the model's norms have one weight for all coordinates
    embed_norm: bool = False       # the stream starts from a normalised embedding
    input_conv: int = 0            # mixers read h + a causal convolution of h over this many tokens, 0: h
    residual_mult: float = 1.0     # x <- x + residual_mult * sublayer
    token_side: int = 0            # width of the per-layer token input, 0: none
    norm_offset: float = 0.0       # added to every stored norm weight
    tied_head: bool = False        # the embedding table is the output matrix
    logit_softcap: float = 0.0     # logits <- cap tanh(logits / cap); 0: none
    extras: dict = field(default_factory=dict)

    def __post_init__(self):
        _positive(self, "vocab_size", "hidden_size", "max_seq_len")
        if self.input_conv < 0:
            raise ValueError(f"input convolution over {self.input_conv} tokens")
        if self.parallel and (self.post_norm or not self.pre_norm or self.token_side or self.position_table):
            raise ValueError("sublayers side by side come with a norm in front only, no token input and no position table")
        for i, x in enumerate(self.layers):
            if self.parallel and (x.attention is None and x.latent is None or isinstance(x.mixer, ParallelMixer)
                                  or isinstance(x.mlp, MoeFF)):
                raise ValueError(f"layer {i}: only attention and dense feed-forwards run side by side")
            a = x.latent
            if a is not None and a.kv_from is not None:
                b = self.layers[a.kv_from].latent if 0 <= a.kv_from < i else None
                if b is None or b.kv_from is not None or (b.kv_rank, b.rot_dim, b.rotation) != (a.kv_rank, a.rot_dim, a.rotation):
                    raise ValueError(f"layer {i}: layer {a.kv_from} has no latents of its shape and rotation to share")
            a = x.attention
            if a is None or a.kv_from is None:
                continue
            b = self.layers[a.kv_from].attention if 0 <= a.kv_from < i else None
            if b is None or b.kv_from is not None or (b.kv_heads, b.dim, b.vdim) != (a.kv_heads, a.dim, a.vdim):
                raise ValueError(f"layer {i}: layer {a.kv_from} has no keys and values of its shape to share")

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
        if arch == "Dogozen":
            return cls(layers=[_dogozen_layer(i, x) for i, x in enumerate(d["layers"])],
                       position_table=False, norm_offset=1.0, tied_head=True, logit_softcap=float(d.get("logit_softcap") or 0.0),
                       **common)
        if arch == "Zigivik":
            return cls(layers=[_zigivik_layer(i, x) for i, x in enumerate(d["layers"])], position_table=False, post_norm=False,
                       parallel=True, scalar_norms=True, embed_norm=True, input_conv=int(d["canon"]["taps"]),
                       residual_mult=float(d["residual_mult"]), **common)
        return cls(layers=[_layer_from_dict(i, x, ("gla", "parallel"), "silu") for i, x in enumerate(d["layers"])],
                   embed_scale=float(d["embedding"]["scale"]), logit_scale=float(d["logit_scale"]),
                   max_seq_len=int(d["max_positions"]), **common)

    def to_dict(self) -> dict:
        layer = {"Dogozen": _dogozen_layer_to_dict, "Zigivik": _zigivik_layer_to_dict}.get(self.architecture, _layer_to_dict)
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "layers": [layer(x) for x in self.layers]}
        if self.architecture == "Lebedra":
            d["residual_mult"] = self.residual_mult
            if self.token_side:
                d["token_side"] = {"dim": self.token_side}
        elif self.architecture == "Dogozen":
            if self.logit_softcap:
                d["logit_softcap"] = self.logit_softcap
        elif self.architecture == "Zigivik":
            d.update(residual_mult=self.residual_mult, canon={"taps": self.input_conv})
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
        mixer = LatentAttentionMixer(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                     float(m["scale"]), Rotation(float(rot["base"]), int(rot.get("dims", m["rot_dim"])), layout="pairs"))
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
                 "rot": {"base": m.rotation.base, "dims": m.rot_dim}}
    else:
        mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}
    f = x.mlp
    if isinstance(f, MoeFF):
        mlp = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit},
               "router": {"experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}
    else:
        mlp = {"kind": "dense", "ff": f.ff} if f is not None else None
    return {"type": x.type, "mixer": mixer, "mlp": mlp}


# ---- Dogozen
def _dogozen_attention(a: dict, **fixed) -> AttentionMixer:
    rot, temp = a.get("rot"), a.get("q_temp")
    scaling = rot.get("scaling") if rot else None
    return AttentionMixer(
        int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
        rotation=Rotation(float(rot["base"]), int(rot["dims"]),
                          FrequencyScaling(*(float(scaling[n]) for n in ("factor", "low", "high", "original"))) if scaling else None)
        if rot else None,
        window=int((a.get("mask") or {}).get("size", 0)),
        q_temp=QueryTemperature(float(temp["coef"]), float(temp["every"])) if temp else None,
        kv_from=int(a["kv_from"]) if a.get("kv_from") is not None else None, **fixed)


def _dogozen_layer(index: int, d: dict) -> LayerSpec:
    kind, m, mlp = d["type"], d["mixer"], d.get("mlp")
    if kind == "attention":
        mixer = _dogozen_attention(m, qk_norm="plain", gate="channel", bias=True)
    elif kind == "parallel":
        r = m["right"]
        mixer = ParallelMixer(_dogozen_attention(m["left"], qk_norm=None, gate=None, sink="learned"),
                              SelectiveMixer(int(r["inner"]), int(r["state"]), int(r["dt_rank"]), int(r["conv"])),
                              (float(m["left_scale"]), float(m["right_scale"])))
    else:
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    if mlp is not None and mlp.get("kind") == "moe":
        r, shared = mlp["router"], mlp.get("shared")
        g = r.get("groups") or {"count": 1, "keep": 1}
        ff = MoeFF(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), groups=int(g["count"]), keep=int(g["keep"]), act="silu",
                   score="sigmoid", correction=False, group_best=2, normalise=True, scale=float(r["scale"]),
                   shared=int(shared["ff"]) if shared else 0)
        return LayerSpec(kind, mixer, ff)
    return LayerSpec(kind, mixer, _mlp_from_dict(index, mlp, "silu"))


def _dogozen_layer_to_dict(x: LayerSpec) -> dict:
    def attention(a: AttentionMixer) -> dict:
        d = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
        if a.rotation:
            d["rot"] = {"base": a.rotation.base, "dims": a.rotation.dims}
            if a.rotation.scaling:
                d["rot"]["scaling"] = dict(vars(a.rotation.scaling))
        if a.window:
            d["mask"] = {"size": a.window}
        if a.q_temp:
            d["q_temp"] = dict(vars(a.q_temp))
        if a.kv_from is not None:
            d["kv_from"] = a.kv_from
        return d

    m, f = x.mixer, x.mlp
    if isinstance(m, ParallelMixer):
        mixer = {"left": attention(m.left), "right": dict(vars(m.right)), "left_scale": m.scales[0], "right_scale": m.scales[1]}
    else:
        mixer = attention(m)
    mlp = {"kind": "dense", "ff": f.ff} if f is not None else None
    if isinstance(f, MoeFF):
        mlp = {"kind": "moe", "expert": {"ff": f.ff},
               "router": {"experts": f.experts, "top": f.top, "scale": f.scale, "groups": {"count": f.groups, "keep": f.keep}}}
        if f.shared:
            mlp["shared"] = {"ff": f.shared}
    return {"type": x.type, "mixer": mixer, "mlp": mlp}


# ---- Zigivik
def _zigivik_layer(index: int, d: dict) -> LayerSpec:
    kind, m, mlp = d["type"], d["mixer"], d.get("mlp")
    if kind not in ("attention", "latent_attention"):
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    rot = m["rot"]
    scaling = rot.get("scaling")
    if scaling:
        scaling = RampScaling(*(float(scaling[n]) for n in ("factor", "original", "fast", "slow")))
    rotation = Rotation(float(rot["base"]), int(rot["dims"]), scaling or None, "pairs" if kind == "attention" else "halves")
    window = int((m.get("mask") or {}).get("size", 0))
    if kind == "attention":
        mixer = AttentionMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), qk_norm=None,
                               gate=None, bias=True, values="keys", rotation=rotation, window=window, sink="zero")
    else:
        mixer = LatentAttentionMixer(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                     float(m["scale"]), rotation, q_rank=int(m["q_rank"]), window=window, sink=None, gate=True,
                                     kv_from=int(m["kv_from"]) if m.get("kv_from") is not None else None)
        _positive(mixer, "q_rank")
    return LayerSpec(kind, mixer, _mlp_from_dict(index, mlp, "poly_norm"))


def _zigivik_layer_to_dict(x: LayerSpec) -> dict:
    m = x.mixer
    r = m.rotation
    rot = {"base": r.base, "dims": r.dims}
    if r.scaling:
        rot["scaling"] = dict(vars(r.scaling))
    mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": rot}
    if isinstance(m, AttentionMixer):
        mixer["kv_heads"] = m.kv_heads
    else:
        mixer.update(rot_dim=m.rot_dim, kv_rank=m.kv_rank, q_rank=m.q_rank)
        if m.kv_from is not None:
            mixer["kv_from"] = m.kv_from
    if m.window:
        mixer["mask"] = {"size": m.window}
    return {"type": x.type, "mixer": mixer, "mlp": {"kind": "dense", "ff": x.mlp.ff} if x.mlp is not None else None}


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
    mixer = LatentAttentionMixer(width // 128, 128, 64, 128, 512, 192 ** -0.5,
                                 Rotation(10000.0, 64, layout="pairs"))
    dense = width * 11 // 4 // 128 * 128
    moe = MoeFF(experts, top, max(128, dense // top // 128 * 128), 7.0, 8, 3)
    out = [LayerSpec("latent_attention", mixer, DenseFF(dense, "relu") if i == 0 else moe) for i in range(layers)]
    return HybridConfig(vocab, width, out, 1e-6, max_seq_len=max_positions, architecture="Lebedra", position_table=False,
                        pre_norm=False, residual_mult=0.5, token_side=128)


def dogozen_config(width: int = 2048, layers: int = 8, vocab: int = 32000, max_positions: int = 8192, experts: int = 64,
                   top: int = 6, window: int = 1024) -> HybridConfig:
    """Dogozen at the layer sizes of a real model: full attention and window attention beside a selective scan of
    twice the width alternate; dense feed-forwards and experts whose ``top`` and shared one together are about as
    wide. The last full-attention layer uses the keys and values of the one before."""
    h = width // 128
    dense = width * 11 // 4 // 128 * 128
    one = max(128, dense // (top + 2) // 128 * 128)
    moe = MoeFF(experts, top, one, groups=8, keep=4, act="silu", score="sigmoid", correction=False, group_best=2, normalise=True,
                scale=2.5, shared=2 * one)
    full = [i for i in range(layers) if i % 2 == 0]
    out = []
    for i in range(layers):
        if i % 2 == 0:
            share = full[-2] if len(full) > 2 and i == full[-1] else None
            out.append(LayerSpec("attention", AttentionMixer(
                h, max(1, h // 8), 128, 128, 128 ** -0.5, qk_norm="plain", gate="channel", bias=True,
                q_temp=QueryTemperature(0.1, 8192), kv_from=share), DenseFF(dense)))
        else:
            out.append(LayerSpec("parallel", ParallelMixer(
                AttentionMixer(h, max(1, h // 8), 128, 128, 128 ** -0.5, qk_norm=None, gate=None, sink="learned", window=window,
                               rotation=Rotation(500000.0, 128, FrequencyScaling(8.0, 1.0, 4.0, 8192))),
                SelectiveMixer(2 * width, 16, max(8, width // 16), 4), (1.0, 1.0)), moe))
    return HybridConfig(vocab, width, out, 1e-6, max_seq_len=max_positions, architecture="Dogozen", position_table=False,
                        norm_offset=1.0, tied_head=True, logit_softcap=50.0)


def zigivik_config(width: int = 2048, layers: int = 8, vocab: int = 32000, max_positions: int = 8192,
                   window: int = 1024) -> HybridConfig:
    """Zigivik at the layer sizes of a real model: every fourth layer full attention (one key head for eight query
    heads, 128 wide), the others window attention over latents of 512 with heads of 128 + 64 rotated; the second of
    three neighbours uses the first one's latents. The ungated feed-forward is as wide as a gated one is in all."""
    h = width // 128
    ff = DenseFF(width * 11 // 4 // 128 * 128 * 3 // 2 // 128 * 128, "poly_norm")
    rot = Rotation(500000.0, 64, RampScaling(8.0, 8192, 32.0, 1.0), "halves")
    out = []
    for i in range(layers):
        if i % 4 == 3:
            out.append(LayerSpec("attention", AttentionMixer(
                h, max(1, h // 8), 128, 128, 128 ** -0.5, qk_norm=None, gate=None, bias=True, values="keys",
                rotation=Rotation(500000.0, 128, layout="pairs"), sink="zero"), ff))
        else:
            out.append(LayerSpec("latent_attention", LatentAttentionMixer(
                h, 128, 64, 128, 512, 192 ** -0.5, rot, q_rank=max(128, width * 3 // 8 // 128 * 128), window=window, sink=None, gate=True,
                kv_from=i - 1 if i % 4 == 1 else None), ff))
    return HybridConfig(vocab, width, out, 1e-6, max_seq_len=max_positions, architecture="Zigivik", position_table=False,
                        post_norm=False, parallel=True, scalar_norms=True, embed_norm=True, input_conv=4, residual_mult=0.7)


register("Dogozen", HybridConfig.from_dict, "mythos_b200.models.hybrid:HybridModel")
register("Lebedra", HybridConfig.from_dict, "mythos_b200.models.hybrid:HybridModel")
register("Teganex", HybridConfig.from_dict, "mythos_b200.models.hybrid:HybridModel")
register("Zigivik", HybridConfig.from_dict, "mythos_b200.models.hybrid:HybridModel")

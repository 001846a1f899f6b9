"""Small layer-list configurations and weights for the hybrid tests."""
import torch

from mythos_b200.models.hybrid import HybridModel, expected_shapes
from mythos_b200.models.hybrid_config import HybridConfig


def attention(heads, kv, dim, vdim, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def gla_layer(heads, dim, vdim, tau, ff=0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel_layer(left, right, ff=0):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, eps=1e-5, embed_scale=1.5, logit_scale=0.7, max_positions=640):
    return {"architecture": "Teganex", "vocab": vocab, "width": width, "max_positions": max_positions,
            "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


def latent(heads, dim, rot, vdim, rank, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": base, "dims": rot},
            "scale": (dim + rot) ** -0.5 if scale is None else scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, groups=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


def lebedra(width, vocab, layers, side, mult=0.5, eps=1e-5):
    return {"architecture": "Lebedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "token_side": {"dim": side},
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


CONFIGS = {
    # unaligned widths everywhere, grouped heads, three taps
    "ragged": config(100, 211, [gla_layer(3, 24, 40, 8.0, ff=52),
                                parallel_layer(attention(6, 2, 20, 36), delta(4, 2, 44, 28, 3)),
                                gla_layer(1, 40, 24, 2.0)]),
    # widths of the tensor-core paths; more than eight query heads on one key head
    "wide": config(256, 384, [parallel_layer(attention(12, 1, 128, 64, 0.11), delta(2, 2, 128, 128, 4), ff=256),
                              gla_layer(2, 128, 80, 16.0, ff=128)]),
    # one head everywhere, one tap, equal key and value widths, no layer with grouped heads
    "single": config(64, 96, [parallel_layer(attention(1, 1, 64, 64), delta(1, 1, 32, 32, 1), ff=64),
                              gla_layer(1, 64, 64, 1.0)], eps=1e-3, embed_scale=1.0, logit_scale=1.0),
    # attention first and last, key wider than value, kv heads between 1 and heads
    "deep": config(128, 160, [parallel_layer(attention(4, 2, 64, 128), delta(6, 3, 64, 48, 2), ff=96),
                              gla_layer(5, 16, 32, 32.0), gla_layer(2, 96, 96, 4.0, ff=72),
                              parallel_layer(attention(8, 4, 128, 128), delta(3, 1, 96, 64, 5))], eps=1e-6),
    # Lebedra: unaligned widths, layers of different sizes, a layer without feed-forward
    "latent_ragged": lebedra(100, 211, [(latent(3, 20, 6, 36, 44), dense(52)), (latent(5, 12, 10, 20, 28, 500.0, 0.3), moe(6, 3, 20, 0.7, 3, 2)),
                                        (latent(2, 40, 14, 12, 60), None)], 12, 0.7),
    # widths of the tensor-core paths, more than 16 heads, no groups
    "latent_wide": lebedra(256, 384, [(latent(20, 128, 64, 128, 256), moe(8, 2, 64, 5.0)), (latent(2, 64, 32, 64, 512), dense(256)),
                                      (latent(4, 72, 40, 104, 128), moe(12, 4, 72, 1.5, 4, 2))], 32, 0.4),
    # one head, one expert, the narrowest rotation, whole residuals
    "latent_single": lebedra(64, 96, [(latent(1, 64, 2, 64, 64, 100.0), moe(1, 1, 64, 2.0)), (latent(1, 24, 8, 40, 40), moe(4, 1, 32, 1.0, 4, 1))],
                             8, 1.0, 1e-3),
    # widths beyond the prompt attention's, a token side wider than a tile
    "latent_plain": lebedra(136, 130, [(latent(2, 160, 72, 136, 40), moe(9, 5, 24, 3.0, 3, 3)), (latent(17, 16, 4, 24, 520), dense(40))], 136, 0.6),
}
TEGANEX = [n for n in CONFIGS if not n.startswith("latent")]
LEBEDRA = [n for n in CONFIGS if n.startswith("latent")]


def weights(cfg: dict, seed: int = 0, low_rank: int = 12, sure_routes: bool = False) -> dict:
    """Random bf16 weights with visible effects: decays from nearly one to nearly zero, write strengths and
    gates spread over their range, norm weights away from one.

    ``sure_routes``: routers read only the first columns of the stream and no sublayer writes those, so that the
    choice of experts depends on the token alone and rounding in bf16 cannot change it."""
    g = torch.Generator().manual_seed(seed)
    hc = HybridConfig.from_dict(cfg)
    out = {}
    for name, shape in expected_shapes(hc).items():
        shape = tuple(low_rank if n is None else n for n in shape)
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if len(shape) == 1:
            if leaf == "A_log":
                t = torch.linspace(-3.0, 2.7, shape[0]) if shape[0] > 1 else torch.zeros(1)
            elif leaf == "dt_bias":
                t = r * 1.5 - 1.0
            elif leaf == "sink":
                t = r * 1.5
            elif leaf == "correction":
                t = r * 0.15
            elif leaf == "b":
                t = r + 2.0
            else:
                t = 1.0 + 0.3 * r
        elif leaf == "conv":
            t = r * 0.5
        elif leaf in ("q", "router") and cfg["architecture"] == "Lebedra":
            t = r * ((1.0 if leaf == "q" else 2.0) / shape[1] ** 0.5)
        elif leaf in ("embed", "pos"):
            t = r * (1.0 if leaf == "embed" else 0.4)
        else:
            t = r * (1.5 / shape[1] ** 0.5)
        if sure_routes and cfg["architecture"] == "Lebedra":
            n = max([x["mlp"]["router"]["experts"] for x in cfg["layers"] if (x["mlp"] or {}).get("kind") == "moe"] or [0])
            if leaf == "router":
                t = torch.cat([r[:, :n] * 2.0 / n ** 0.5, torch.zeros(shape[0], shape[1] - n)], 1)
            elif leaf in ("o", "down", "proj"):
                t[:n] = 0.0
        out[name] = t.to(torch.bfloat16)
    return out


def model(cfg: dict, seed: int = 0, device="cuda", w=None) -> HybridModel:
    return HybridModel(HybridConfig.from_dict(cfg), dict(w if w is not None else weights(cfg, seed))).to(device)


def tokens(cfg: dict, n: int, seed: int = 1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(a, b, scale=None):
    """Root-mean-square error of every row relative to the rms of the reference (or of ``scale``)."""
    a, b = a.double().cpu(), b.double().cpu()
    return (a - b).pow(2).mean(-1).sqrt() / (b if scale is None else scale).double().pow(2).mean().sqrt()


def rel(a, b):
    """Largest root-mean-square error of a row relative to the rms of the reference."""
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).pow(2).mean(-1).sqrt().max() / b.pow(2).mean().sqrt())

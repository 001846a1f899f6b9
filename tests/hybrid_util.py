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


def window_left(heads, kv, dim, vdim, rot, window, base=500.0, scaling=None, scale=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "rot": r,
            "mask": {"size": window}}


def selective(inner, state, rank, conv):
    return {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}


def tempered_layer(heads, kv, dim, vdim, coef, every, scale=None, mlp=None, kv_from=None):
    m = dict(attention(heads, kv, dim, vdim, scale), q_temp={"coef": coef, "every": every})
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def scan_layer(left, right, scales, mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def sigmoid_moe(experts, top, ff, groups, keep, scale=1.0, shared=0):
    d = {"kind": "moe", "expert": {"ff": ff},
         "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def dogozen(width, vocab, layers, cap=20.0, eps=1e-5):
    return {"architecture": "Dogozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


def ramp(base, dims, factor=None, original=64, fast=8.0, slow=1.0):
    """Rotation with slowed long wavelengths (without, where ``factor`` is None)."""
    r = {"base": base, "dims": dims}
    if factor is not None:
        r["scaling"] = {"factor": factor, "original": float(original), "fast": fast, "slow": slow}
    return r


def window_latent(heads, dim, rot, vdim, rank, q_rank, window, turn=None, scale=None, kv_from=None, ff=0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "mask": {"size": window},
         "rot": turn or ramp(300.0, rot), "scale": (dim + rot) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": dense(ff) if ff else None}


def key_value(heads, kv, dim, rot, base=400.0, scale=None, ff=0):
    m = dict(attention(heads, kv, dim, dim, scale), rot={"base": base, "dims": rot})
    return {"type": "attention", "mixer": m, "mlp": dense(ff) if ff else None}


def zigivik(width, vocab, layers, taps, mult, eps=1e-5):
    return {"architecture": "Zigivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "canon": {"taps": taps},
            "layers": layers}


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
    # Dogozen: unaligned widths, shared keys and values with another temperature and scale, partial rotation of an odd
    # number of pairs, three taps, fewer channels than a block
    "scan_ragged": dogozen(100, 211, [
        tempered_layer(6, 2, 20, 36, 0.4, 16, mlp=dense(52)),
        scan_layer(window_left(4, 2, 20, 12, 10, 19), selective(52, 5, 3, 3), (0.7, 1.2), sigmoid_moe(6, 3, 20, 3, 2, 1.7, 28)),
        tempered_layer(4, 2, 20, 36, 0.9, 7, 0.4, kv_from=0)]),
    # widths of the tensor-core paths, more than eight query heads on one key head, stretched rotation, two lanes per
    # channel, a layer that shares with the one before a parallel layer
    "scan_wide": dogozen(256, 384, [
        scan_layer(window_left(6, 2, 72, 104, 48, 70, 1e4, (4.0, 1.0, 3.0, 64)), selective(512, 16, 16, 4), (1.0, 0.6), dense(256)),
        tempered_layer(12, 1, 128, 64, 0.2, 100, 0.11, sigmoid_moe(8, 2, 64, 2, 1, 2.0, 64)),
        scan_layer(window_left(4, 4, 128, 128, 128, 33, 1e5, (8.0, 1.0, 4.0, 512)), selective(200, 24, 40, 4), (0.5, 0.9),
                   sigmoid_moe(12, 4, 72, 1, 1)),
        tempered_layer(9, 1, 128, 64, 0.3, 1, 0.09, dense(96), kv_from=1)], 18.0),
    # one of everything: head, tap, state value, rank, window, expert, experts per group
    "scan_single": dogozen(64, 96, [
        scan_layer(window_left(1, 1, 16, 16, 2, 1), selective(8, 1, 1, 1), (1.0, 1.0), sigmoid_moe(4, 1, 24, 4, 2, 0.5, 8)),
        tempered_layer(1, 1, 64, 64, 1.5, 3, mlp=sigmoid_moe(1, 1, 32, 1, 1)),
        scan_layer(window_left(2, 1, 64, 64, 64, 16), selective(72, 4, 9, 2), (2.0, -0.5))], 50.0, 1e-3),
    # widths beyond the prompt attention's, a window longer than the sequences, many state values, many taps
    "scan_plain": dogozen(136, 130, [
        tempered_layer(2, 2, 160, 136, 0.5, 32, mlp=dense(40)),
        scan_layer(window_left(3, 1, 136, 24, 40, 2000), selective(40, 130, 24, 6), (0.9, 1.1), dense(56))], 10.0),
    # Zigivik: unaligned widths, grouped heads, partial rotation of an odd number of pairs, three taps, a layer without
    # feed-forward, latents shared with other heads, another window and scale
    "side_ragged": zigivik(100, 211, [
        window_latent(3, 20, 6, 36, 44, 28, 19, ramp(300.0, 6, 4.0), ff=52),
        key_value(6, 2, 20, 10, ff=44),
        window_latent(5, 12, 6, 20, 44, 21, 33, ramp(300.0, 6, 4.0), 0.35, kv_from=0),
        key_value(3, 3, 28, 28, scale=0.3)], 3, 0.55),
    # widths of the tensor-core paths, more than 16 latent heads, more than eight query heads on one key head, a window
    # longer than a key tile, the sharing layer behind another that has latents of its own
    "side_wide": zigivik(256, 384, [
        key_value(12, 1, 128, 128, 1e4, 0.11, ff=512),
        window_latent(20, 128, 64, 128, 256, 136, 70, ramp(1e4, 64, 8.0, 128, 32.0), ff=256),
        window_latent(2, 64, 32, 64, 512, 64, 100, ramp(500.0, 32), ff=264),
        window_latent(4, 72, 64, 104, 256, 80, 64, ramp(1e4, 64, 8.0, 128, 32.0), kv_from=1, ff=328),
        key_value(4, 4, 64, 48, 1e5, ff=128)], 4, 0.4),
    # one head, pair, tap, key and rank; whole residuals; every layer narrow
    "side_single": zigivik(64, 96, [
        window_latent(1, 16, 2, 16, 8, 1, 1, ramp(100.0, 2, 2.0, 16, 2.0, 1.0), ff=1),
        key_value(1, 1, 64, 2, 10.0, ff=64),
        window_latent(1, 8, 8, 8, 16, 64, 16, ff=8)], 1, 1.0, 1e-3),
    # widths beyond the prompt attention's, latents beyond the decode kernel's, a window longer than the sequences, many taps
    "side_plain": zigivik(136, 130, [
        window_latent(2, 160, 72, 136, 40, 136, 2000, ramp(1e4, 72, 16.0, 32, 4.0, 0.5), ff=40),
        key_value(2, 1, 136, 72, ff=2100),
        window_latent(3, 16, 4, 24, 520, 30, 40, ff=24)], 6, 0.6),
}
TEGANEX = [n for n in CONFIGS if not n.startswith(("latent", "scan", "side"))]
LEBEDRA = [n for n in CONFIGS if n.startswith("latent")]
DOGOZEN = [n for n in CONFIGS if n.startswith("scan")]
ZIGIVIK = [n for n in CONFIGS if n.startswith("side")]


def _zigivik_weight(name: str, r: torch.Tensor) -> torch.Tensor:
    """Norm weights away from one, every power of the activation and every bias and tap visible."""
    leaf = name.rsplit(".", 1)[-1]
    if leaf == "act":
        return torch.tensor([0.7, -0.5, 0.4, 0.3]) + 0.1 * r
    if len(r.shape) == 0 or leaf == "norm":
        return 1.0 + 0.3 * r
    if len(r.shape) == 1:
        return 0.5 * r
    if leaf == "canon1":
        return 0.4 * r
    return r if leaf == "embed" else r * (1.5 / r.shape[1] ** 0.5)


def _dogozen_weight(name: str, r: torch.Tensor) -> torch.Tensor:
    """Norms around zero, decays from nearly one to nearly zero, biases and step sizes that show."""
    leaf = name.rsplit(".", 1)[-1]
    if leaf == "A_log":
        return r * 1.2 - 0.5
    if len(r.shape) == 1:
        if name.endswith(".dt.b"):
            return r * 1.5 - 2.0
        return 1.0 + 0.3 * r if leaf == "D" else r * {"sink": 1.5, "b": 0.5}.get(leaf, 0.3)
    if leaf == "conv":
        return r * 0.5
    if leaf == "embed":
        return r
    return r * ({"router": 2.0, "dt": 1.0}.get(leaf, 1.5) / r.shape[1] ** 0.5)


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
        if cfg["architecture"] in ("Dogozen", "Zigivik"):
            t = {"Dogozen": _dogozen_weight, "Zigivik": _zigivik_weight}[cfg["architecture"]](name, r)
        elif len(shape) == 1:
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
        if sure_routes and cfg["architecture"] != "Teganex":
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

"""Tiny Lovapel configurations for the tests and the plain implementation's logits for them.

The configurations differ from one another in every size and option: widths, head counts and grouping (one key/value
head per query head, one for all, some), key size against value size, windows shorter than a page, longer than several
pages, and absent, rotation over part of a head, over all of it, and absent, layers without a feed-forward, routers with
and without groups (of several experts and of one), identity experts (none, few, more than real ones), shared experts
(absent, smaller and larger than the routed ones), every expert chosen / one chosen, spans run several times (at the
start, in the middle, at the end, none), logit scales and caps present and absent, sizes the tensor-core kernels take and
sizes that are multiples of nothing convenient.  Pages of 4, 8, 16 and 32 tokens.

A router's choice jumps where two choice scores meet, and in bfloat16 some token of some layer always stands there.  The
bfloat16 runs therefore use the same models with corrections that lie far apart (`separate_corrections`), so that
rounding moves weights but not choices; the 32-bit runs use the random corrections, and choose differently for every token."""
import os

import torch

import plain_lovapel as pl


def attention(heads, kv, dim, vdim, scale, window=None, rot=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=None, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, eps, init, layers, loop=None, scale=None, cap=None):
    d = {"architecture": "Lovapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "initializer_range": init, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    if scale is not None:
        d["logit_scale"] = scale
    if cap is not None:
        d["logit_softcap"] = cap
    return d


# sizes the bfloat16 tensor-core kernels take (keys and values in multiples of 16, widths in multiples of 8)
LOV_A = model(211, 64, 1e-5, 0.1, [
    attention(4, 2, 16, 32, 0.3, 20, (8, 100.0), dense(96)),
    attention(4, 1, 32, 16, 0.2, 37, (32, 5000.0), moe(10, 3, 40, identity=2, groups=(3, 2), shared=24)),
    attention(6, 6, 16, 16, 0.35, None, (4, 30.0), moe(7, 2, 56, identity=1, groups=(4, 2))),
], loop=(1, 3, 2), scale=1.5, cap=8.0)
# sizes that are multiples of nothing convenient; a window shorter than the page; one expert chosen; a layer three times
LOV_B = model(128, 44, 1e-4, 0.15, [
    attention(6, 3, 10, 6, 0.5, 3, (10, 30.0), moe(7, 1, 12)),
    attention(2, 1, 6, 18, 0.4, 41, (2, 10.0)),
    attention(5, 5, 7, 9, 0.6, 9, (6, 1000.0), moe(3, 2, 10, identity=6, groups=(3, 2), shared=22)),
], loop=(2, 3, 3), scale=0.7, cap=3.0)
# no span, no window, no rotation, no cap; groups of one; more identity experts than real ones; everything chosen
LOV_C = model(97, 40, 1e-6, 0.12, [
    attention(5, 1, 8, 8, 0.4, None, None, moe(5, 5, 16, identity=3, groups=(8, 5), shared=8)),
    attention(3, 3, 20, 12, 0.3, 17, None, moe(2, 6, 24, identity=4)),
    attention(4, 2, 8, 16, 0.5, None, (6, 50.0), dense(28)),
])
# larger: head groups of 8, windows of hundreds over many pages, gate and up blocks of 128, a span at the start
LOV_D = model(257, 128, 1e-6, 0.05, [
    attention(8, 1, 64, 32, 0.18, 150, (32, 10000.0), moe(14, 2, 128, identity=2, groups=(4, 1), shared=160)),
    attention(16, 4, 16, 64, 0.25, 65, (16, 500.0), dense(256)),
    attention(8, 2, 32, 48, 0.12, 129, (24, 250000.0), moe(12, 4, 256, identity=4, groups=(2, 2), shared=128)),
    attention(2, 2, 128, 128, 0.09, None, (64, 2000.0)),
], loop=(0, 2, 2), cap=20.0)
LOV = {"A": (LOV_A, 16, 3), "B": (LOV_B, 4, 4), "C": (LOV_C, 8, 5), "D": (LOV_D, 32, 9)}   # config, page size, seed


def separate_corrections(weights, seed):
    """Corrections in random order, 1.5 apart (softmax scores lie within 1 of each other): every token of a layer takes
    the same experts, with weights of its own."""
    g = torch.Generator().manual_seed(seed)
    for name in sorted(weights):
        if name.endswith(".correction"):
            n = weights[name].numel()
            weights[name] = (torch.randperm(n, generator=g).float() - n / 2) * 1.5
    return weights


def write_models(tmp_path_factory):
    """Two folders per configuration, by the dtype they are run in."""
    from tiny_llm_b200.config import LovapelConfig
    from tiny_llm_b200.weights import write_random_model
    from tiny_llm_b200.weights.safetensors_io import save_safetensors

    out = {}
    for name, (cfg, _page, seed) in LOV.items():
        out[name] = {}
        for dtype in ("float32", "bfloat16"):
            d = str(tmp_path_factory.mktemp(f"lov_{name}_{dtype}"))
            write_random_model(d, LovapelConfig.from_dict(cfg), seed=seed, dtype=torch.float32)
            if dtype == "bfloat16":
                save_safetensors(os.path.join(d, "model.safetensors"), separate_corrections(pl.load_weights(d), seed))
            out[name][dtype] = d
    return out


def plain_model(model_dir, dtype):
    """Configuration, weights and storage rounding of the plain implementation for one of the engine's two paths."""
    cfg, w = pl.load_config(model_dir), pl.load_weights(model_dir)
    if dtype == "bfloat16":   # matrices are held in the engine's dtype, vectors in 32-bit
        w = {k: (v if v.dim() < 2 else v.to(torch.bfloat16).float()) for k, v in w.items()}
    return cfg, w, (pl.no_quant if dtype == "float32" else pl.bf16_quant)


def plain_logits(model_dir, reqs, dtype):
    """What the engine's logits are held against: the plain implementation in 64-bit with the path's weights (rounded
    to bfloat16 for the bfloat16 path) and NO rounding of activations, i.e. the result the path approximates."""
    cfg, w, _ = plain_model(model_dir, dtype)
    return {rid: pl.forward(cfg, w, toks, torch.float64).float() for rid, toks in reqs.items()}


def tolerances(model_dir, reqs, dtype):
    """Per request, how far the engine may be from the plain implementation's 64-bit logits.  32-bit: 2e-5, or four
    times what 32-bit rounding does to the plain implementation itself where that is more.  bfloat16: twice what
    bfloat16 rounding of the activations does to the plain implementation for this very request.  The engine rounds
    at the same places but sums in another order, so its error is another draw of the same size.  (A fault -- a
    wrong key, a lost state, a window edge off by one -- is caught by the 32-bit runs of the same code.)"""
    out = {}
    for rid, toks in reqs.items():
        cfg, w, quant = plain_model(model_dir, dtype)
        f64 = pl.forward(cfg, w, toks, torch.float64)
        if dtype == "float32":
            f32 = pl.forward(cfg, w, toks, torch.float32)
            out[rid] = max(2e-5, 4.0 * float((f32.double() - f64).abs().max()))
        else:
            out[rid] = 2.0 * float((pl.forward(cfg, w, toks, torch.float64, quant=quant) - f64).abs().max())
    return out


def compare(got, ref, prefix, tol, what):
    worst = 0.0
    for rid, r in ref.items():
        g = got[prefix + rid]
        assert g.shape == r.shape, (what, rid, g.shape, r.shape)
        diff = (g - r).abs()
        if not float(diff.max()) <= tol[rid]:
            bad = (~(diff.max(dim=1).values <= tol[rid])).nonzero().flatten()
            raise AssertionError(f"{what}: request {rid} differs from the plain implementation first at position "
                                 f"{int(bad[0])} of {r.shape[0]} (max |diff| {float(diff.max()):.3e}, tolerance "
                                 f"{tol[rid]:.3e}; wrong positions: {bad.tolist()[:20]})")
        worst = max(worst, float(diff.max()) / tol[rid])
    import replay_util
    replay_util.record_margin(what, "", worst)   # printed, and appended to the file TLLM_MARGIN_FILE names
    return worst

"""Tiny Vigodra configurations for the tests and the plain implementation's logits for them.

The configurations differ from one another in every size and option: widths, head counts and grouping (one key/value
head per query head, one for all, some), key size against value size, filters of 1 to 6 taps, windows shorter than a page,
longer than several pages, and absent, first positions that a window keeps (none, fewer than a page, several pages, more
than the window), distance biases whose last bucket begins inside and far behind the window, rotation over the whole
rotated part and over part of it, a latent layer that reads another layer's cache with a longer or a shorter window than
its owner's, or with none (directly behind it, and several layers on, twice), layers without a feed-forward, limits that
bind always and never, an embedding scale and a stream factor of 1, one mixer only, sizes the tensor-core kernels take and
sizes that are multiples of nothing convenient.  Pages of 4, 8, 16 and 32 tokens."""
import torch

import plain_vigodra as pv


def attention(heads, kv, dim, vdim, scale, conv, far, window=None, keep=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "bias_max": far}
    if window:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, rank, scale, dims, base, window=None, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"dims": dims, "base": base}}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def model(vocab, width, scale, alpha, eps, init, layers):
    return {"architecture": "Vigodra", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "postln_alpha": alpha, "initializer_range": init, "layers": layers}


# sizes the bfloat16 tensor-core kernels take (keys and values in multiples of 16, widths in multiples of 8); the reader of
# the shared latents sees farther back than their owner
VIG_A = model(211, 64, 8.0, 1.7, 1e-5, 0.1, [
    attention(4, 2, 16, 32, 0.3, 4, 37, window=20, keep=5, mlp=dense(96, 0.4)),
    latent(3, 16, 16, 32, 32, 0.25, 16, 100.0, window=24, mlp=dense(72, 5.0)),
    attention(4, 1, 32, 16, 0.2, 3, 64, window=33, keep=40),
    latent(2, 32, 16, 16, 32, 0.2, 16, 100.0, window=50, kv_from=1, mlp=dense(40, 0.1)),
])
# sizes that are multiples of nothing convenient; a window shorter than the page; no window; no kept positions; one tap;
# a reader whose window is shorter than its owner's; a rotation over part of the rotated part
VIG_B = model(128, 44, 1.0, 0.8, 1e-4, 0.15, [
    latent(5, 6, 10, 14, 18, 0.4, 6, 30.0, mlp=dense(20, 1.0)),
    attention(6, 3, 10, 6, 0.5, 2, 9, window=3, keep=2, mlp=dense(28, 0.3)),
    latent(2, 12, 10, 6, 18, 0.3, 6, 30.0, window=7, kv_from=0),
    attention(2, 2, 12, 14, 0.3, 1, 50.5, mlp=dense(12, 2.0)),
    attention(5, 1, 7, 9, 0.6, 6, 130, window=41, keep=0),
    latent(1, 9, 2, 11, 5, 0.7, 2, 10.0, window=5, mlp=dense(16, 0.5)),
])
# one mixer only, no feed-forward anywhere, a stream factor of 1
VIG_C = model(97, 40, 2.0, 1.0, 1e-5, 0.12, [
    attention(5, 5, 8, 8, 0.4, 2, 20, window=9, keep=17),
    attention(2, 1, 20, 12, 0.3, 5, 300),
    attention(4, 2, 8, 16, 0.5, 4, 12, window=100, keep=3),
])
# larger: head groups of 8 and 4, windows of hundreds over many pages, kept positions over several pages, two layers
# reading one layer's cache (one of them without a window), seven layers
VIG_D = model(257, 128, 11.3, 2.4, 1e-6, 0.05, [
    attention(8, 1, 32, 64, 0.18, 4, 90, window=150, keep=70, mlp=dense(160, 0.7)),
    latent(8, 32, 16, 48, 64, 0.15, 16, 10000.0, window=30, mlp=dense(96, 0.5)),
    attention(8, 2, 64, 32, 0.12, 2, 200, window=129, keep=33, mlp=dense(64, 1.1)),
    latent(4, 48, 16, 16, 64, 0.1, 16, 10000.0, kv_from=1, mlp=dense(64, 0.9)),
    latent(2, 16, 32, 80, 48, 0.2, 32, 500.0, window=200),
    latent(2, 16, 16, 80, 64, 0.2, 16, 10000.0, window=129, kv_from=1, mlp=dense(48, 3.0)),
    attention(16, 4, 16, 16, 0.25, 3, 33, window=65, keep=1, mlp=dense(128, 0.2)),
])
VIG = {"A": (VIG_A, 16, 3), "B": (VIG_B, 4, 4), "C": (VIG_C, 8, 5), "D": (VIG_D, 32, 9)}   # config, page size, seed


def write_models(tmp_path_factory):
    from tiny_llm_b200.config import VigodraConfig
    from tiny_llm_b200.weights import write_random_model

    out = {}
    for name, (cfg, _page, seed) in VIG.items():
        d = tmp_path_factory.mktemp(f"vig_{name}")
        write_random_model(str(d), VigodraConfig.from_dict(cfg), seed=seed, dtype=torch.float32)
        out[name] = str(d)
    return out


def plain_model(model_dir, dtype):
    """Configuration, weights and storage rounding of the plain implementation for one of the engine's two paths."""
    cfg, w = pv.load_config(model_dir), pv.load_weights(model_dir)
    if dtype == "bfloat16":   # matrices are held in the engine's dtype; vectors, filters and the distance biases in 32-bit
        w = {k: (v if v.dim() < 2 or k.endswith(".conv") or k.endswith(".rel") else v.to(torch.bfloat16).float())
             for k, v in w.items()}
    return cfg, w, (pv.no_quant if dtype == "float32" else pv.bf16_quant)


def plain_logits(model_dir, reqs, dtype):
    """What the engine's logits are held against: the plain implementation in 64-bit with the path's weights (rounded
    to bfloat16 for the bfloat16 path) and NO rounding of activations, i.e. the result the path approximates."""
    cfg, w, _ = plain_model(model_dir, dtype)
    return {rid: pv.forward(cfg, w, toks, torch.float64).float() for rid, toks in reqs.items()}


def tolerances(model_dir, reqs, dtype):
    """Per request, how far the engine may be from the plain implementation's 64-bit logits.  32-bit: 2e-5, or four
    times what 32-bit rounding does to the plain implementation itself where that is more.  bfloat16: twice what
    bfloat16 rounding of the activations does to the plain implementation for this very request.  The engine rounds
    at the same places but sums in another order, so its error is another draw of the same size.  (A fault -- a
    wrong key, a lost state, a window edge off by one -- is caught by the 32-bit runs of the same code.)"""
    out = {}
    for rid, toks in reqs.items():
        cfg, w, quant = plain_model(model_dir, dtype)
        f64 = pv.forward(cfg, w, toks, torch.float64)
        if dtype == "float32":
            f32 = pv.forward(cfg, w, toks, torch.float32)
            out[rid] = max(2e-5, 4.0 * float((f32.double() - f64).abs().max()))
        else:
            out[rid] = 2.0 * float((pv.forward(cfg, w, toks, torch.float64, quant=quant) - f64).abs().max())
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

"""Small Busatar configurations for the tests; scores are scaled so that attention is peaked and single keys matter."""


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _gqa(heads, kv, dim, vdim, window, scale=0.5):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale}


def _latent(heads, dim, rot, vdim, rank, window, scale=0.3, base=10000.0, scaling=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window}, "scale": scale, "rot": r}


def _lru(width, blocks, taps):
    return {"width": width, "blocks": blocks, "conv": taps}


def _glu(ff, limit):
    return {"ff": ff, "kind": "dense", "limit": limit}


def _model(width, vocab, alpha, eps, layers):
    return {"architecture": "Busatar", "width": width, "vocab": vocab, "postln_alpha": alpha, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # every mixer with and without a feed-forward, grouped heads, all sizes different
    "mixed": _model(192, 320, 1.7, 1e-5, [
        _layer("latent_attention", _latent(4, 32, 8, 48, 64, 40, scaling=(4.0, 64, 8.0, 1.0)), _glu(256, 1.5)),
        _layer("attention", _gqa(6, 2, 48, 32, 33), None),
        _layer("rglru", _lru(160, 5, 4), _glu(192, 0.8)),
        _layer("latent_attention", _latent(2, 64, 32, 32, 128, 17, scaling=(2.0, 4096, 32.0, 1.0)), None),
        _layer("rglru", _lru(96, 1, 2), None),
        _layer("attention", _gqa(4, 4, 32, 64, 128), _glu(128, 3.0))]),
    # sizes that are not multiples of the kernels' tiles
    "odd": _model(200, 131, 2.25, 1e-3, [
        _layer("rglru", _lru(120, 3, 3), _glu(100, 2.5)),
        _layer("attention", _gqa(3, 1, 40, 24, 21), _glu(72, 0.5)),
        _layer("latent_attention", _latent(3, 40, 24, 40, 72, 50, base=500.0), _glu(100, 1.0)),
        _layer("rglru", _lru(40, 5, 1), None)]),
    # large heads: the sizes that only some of the tensor-core kernels serve
    "large": _model(256, 512, 1.0, 1e-6, [
        _layer("attention", _gqa(2, 1, 192, 128, 70, scale=0.2), _glu(320, 1.0)),
        _layer("latent_attention", _latent(20, 128, 64, 128, 256, 129, scale=0.1, scaling=(8.0, 256, 16.0, 2.0)), None),
        _layer("latent_attention", _latent(2, 160, 16, 32, 96, 1000, scale=0.1), _glu(64, 1.0)),
        _layer("attention", _gqa(9, 1, 256, 256, 1, scale=0.2), None)]),
    "recurrent": _model(128, 96, 1.3, 1e-5, [_layer("rglru", _lru(128, 4, 4), None), _layer("rglru", _lru(256, 2, 5), _glu(128, 1.2))]),
}

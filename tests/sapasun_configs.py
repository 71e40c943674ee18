"""Small Sapasun configurations for the tests."""


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def _att(heads, kv, dim, vdim, chunk, rot, taps, v_mix=True, scale=0.4, base=10000.0):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": {"base": base, "dims": rot}, "conv": taps, "scale": scale,
            "v_mix": v_mix}


def _delta(heads, kv, dim, vdim, taps):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": taps}


def _model(width, vocab, eps, cap, layers):
    return {"architecture": "Sapasun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


CONFIGS = {
    # both mixers with and without a feed-forward, shared keys, the first layer that mixes values is not the first attention layer
    "mixed": _model(192, 320, 1e-5, 9.0, [
        _layer("attention", _att(6, 3, 32, 48, 40, 16, 4, v_mix=False), 256),
        _layer("channel_delta", _delta(6, 2, 32, 48, 4), 128),
        _layer("attention", _att(6, 2, 48, 32, 33, 24, 2, base=500.0), None),
        _layer("channel_delta", _delta(3, 3, 64, 16, 2), None),
        _layer("attention", _att(4, 2, 64, 32, 128, 64, 3, scale=0.2), 192),
        _layer("attention", _att(2, 1, 80, 64, 17, 8, 1, scale=0.2), None)]),
    # sizes that are not multiples of the kernels' pieces; long filters
    "odd": _model(90, 131, 1e-3, 3.0, [
        _layer("channel_delta", _delta(3, 1, 22, 13, 5), 100),
        _layer("attention", _att(3, 1, 22, 13, 21, 10, 6), 72),
        _layer("attention", _att(5, 1, 27, 13, 7, 6, 3), None),
        _layer("channel_delta", _delta(5, 5, 9, 30, 1), 33)]),
    # large heads: sizes that only some of the kernels serve, heads that several CTAs share
    "large": _model(256, 512, 1e-6, 20.0, [
        _layer("channel_delta", _delta(4, 2, 128, 128, 4), 320),
        _layer("attention", _att(9, 1, 192, 128, 70, 192, 4, scale=0.07), 320),
        _layer("channel_delta", _delta(2, 1, 144, 272, 3), None),
        _layer("attention", _att(2, 2, 256, 64, 1000, 32, 2, scale=0.07), None),
        _layer("channel_delta", _delta(1, 1, 256, 256, 2), 64)]),
    # one mixer only; filters of a single tap, all heads alike, whole heads rotated
    "attention": _model(128, 96, 1e-5, 5.0, [
        _layer("attention", _att(4, 4, 32, 32, 48, 32, 1, v_mix=False), 128),
        _layer("attention", _att(4, 1, 32, 32, 1, 32, 3, v_mix=False), 128)]),
    "recurrent": _model(128, 96, 1e-5, 5.0, [_layer("channel_delta", _delta(4, 4, 32, 32, 1), None), _layer("channel_delta", _delta(8, 2, 16, 16, 4), 128)]),
}

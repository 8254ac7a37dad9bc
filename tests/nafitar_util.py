"""Small Nafitar configurations for the tests."""
from tests.plan_util import assert_close, make_engine, make_rows, rms_error, run_alone, run_mixed, tokens  # noqa: F401


def layer_conf(heads, kv_heads, dim, window, scale, mem_heads, mem_dim, mem_vdim, cap, ff):
    return dict(type="parallel", mlp=None if ff is None else dict(ff=ff, kind="dense"), mixer=dict(
        left=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask=dict(size=window), scale=scale),
        right=dict(heads=mem_heads, dim=mem_dim, vdim=mem_vdim, gate_cap=cap)))


def conf(layers, width, vocab, loop=None, positions=512, eps=1e-5):
    c = dict(architecture="Nafitar", layers=layers, max_positions=positions, norm=dict(eps=eps), vocab=vocab, width=width)
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def uneven_conf(positions=512):
    """Layers that share no size, odd widths everywhere, one layer without a feed-forward, a loop in the middle."""
    return conf([layer_conf(6, 3, 20, 37, 0.3, 3, 12, 20, 5.0, 36), layer_conf(4, 1, 16, 5, 0.2, 2, 8, 24, 9.0, None),
                 layer_conf(2, 2, 24, 2, 0.25, 1, 40, 70, 3.0, 44)], width=44, vocab=75, loop=(1, 3, 3), positions=positions)


def round_conf(window=70, loop=(0, 1, 2), positions=1024):
    """Two equal layers with sizes the tensor-core kernels take without padding."""
    return conf([layer_conf(8, 2, 128, window, 0.09, 4, 64, 128, 12.0, 192)] * 2, width=192, vocab=320, loop=loop,
                positions=positions)

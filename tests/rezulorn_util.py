"""Small Rezulorn configurations for the tests."""
from tests import plan_util
from tests.oracle import rezulorn as oracle
from tests.plan_util import make_engine, make_rows, rms_error, run_alone, run_mixed, tokens  # noqa: F401


def rotation(dims, base, factor=None):
    return dict(dims=dims, base=base, **(dict(scaling=dict(factor=factor)) if factor else {}))


def attention(heads, kv_heads, dim, vdim, window, keep, scale, ff):
    return dict(type="attention", mlp=dense(ff), mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
                                                            mask=dict(size=window, keep_first=keep)))


def lightning(heads, dim, vdim, decay, ff):
    return dict(type="lightning", mlp=dense(ff), mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay)))


def gates(heads, kv_heads, dim, vdim, rot, scale):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=rot, scale=scale)


def retention(heads, dim, vdim, rot, decay):
    return dict(heads=heads, dim=dim, vdim=vdim, rot=rot, decay=list(decay))


def parallel(left, right, left_scale, right_scale, ff):
    return dict(type="parallel", mlp=dense(ff), mixer=dict(left=left, right=right, left_scale=left_scale,
                                                           right_scale=right_scale))


def dense(ff):
    return dict(kind="dense", ff=ff) if ff else None


def conf(layers, width, vocab, taps=3, mult=0.8, logits=1.5, eps=1e-5):
    return dict(architecture="Rezulorn", canon=dict(taps=taps), layers=layers, logit_scale=logits, norm=dict(eps=eps),
                residual_mult=mult, vocab=vocab, width=width)


def uneven_conf(taps=4, **kw):
    """Layers that share no size, odd widths everywhere, a rotation with and without scaling, layers without feed-forward."""
    ly = [attention(6, 2, 20, 12, 9, 3, 0.3, 36),
          parallel(gates(3, 1, 12, 28, rotation(6, 90.0, 3.0), 0.4), retention(2, 10, 20, rotation(10, 300.0), [0.9, 0.35]),
                   0.7, 1.3, 52),
          lightning(3, 12, 20, [0.999, 0.5, 0.9], None),
          attention(5, 5, 10, 30, 1, 0, 0.25, None),
          parallel(gates(4, 2, 10, 10, rotation(10, 40.0), 0.5), retention(3, 14, 6, rotation(4, 20.0, 1.7), [0.99, 0.8, 0.97]),
                   1.4, 0.6, None),
          attention(2, 1, 16, 8, 70, 20, 0.3, 20),
          lightning(1, 6, 36, [1.0], 28)]
    return conf(ly, width=44, vocab=75, taps=taps, **kw)


def round_conf(taps=3, **kw):
    """Sizes the tensor-core kernels take without padding."""
    ly = [parallel(gates(8, 2, 64, 64, rotation(64, 500.0, 2.0), 0.25),
                   retention(4, 64, 64, rotation(64, 9000.0), [0.97, 0.999, 0.5, 0.99]), 0.5, 0.9, 512),
          attention(8, 4, 128, 64, 100, 5, 0.09, 384),
          lightning(2, 128, 128, [0.98, 0.9995], 256),
          attention(4, 1, 64, 128, 48, 70, 0.12, None),
          parallel(gates(4, 4, 128, 128, rotation(96, 9000.0), 0.2), retention(2, 32, 128, rotation(16, 500.0), [0.9, 0.995]),
                   1.2, 0.4, 256)]
    return conf(ly, width=256, vocab=320, taps=taps, **kw)


def forward(W, c, seq):
    return oracle.forward(W, c, seq)[0]


def assert_close(got, want, dtype="float32", what=None):
    if dtype == "float32":
        return plan_util.assert_close(got, want, dtype, what)
    e = rms_error(got, want)
    assert e.max() < 0.1 and e.quantile(0.9) < 0.03, (what, float(e.max()), float(e.quantile(0.9)), int(e.argmax()))

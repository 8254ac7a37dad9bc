"""Small Kedesun configurations for the tests."""
from tests.plan_util import assert_close, make_engine, make_rows, rms_error, run_alone, run_mixed, tokens  # noqa: F401


def rotation(dims, base, factor=3.0, original=60, fast=9.0, slow=2.0):
    return dict(dims=dims, base=base, scaling=dict(factor=factor, original=original, fast=fast, slow=slow))


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, mlp, base=500.0, **yarn):
    return dict(type="latent_attention", mlp=mlp, mixer=dict(
        heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=rotation(rot_dim, base, **yarn)))


def retention(heads, dim, vdim, mlp, decay=None):
    decay = decay or [1 - 2.0 ** -(1 + 7 * h / max(1, heads - 1)) for h in range(heads)]
    return dict(type="retention", mlp=mlp, mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=decay))


def dense(ff):
    return dict(kind="dense", ff=ff)


def experts(n, top, ff, shared):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=n, top=top), shared=dict(ff=shared))


def conf(layers, width, vocab, eps=1e-5):
    return dict(architecture="Kedesun", layers=layers, norm=dict(eps=eps), vocab=vocab, width=width)


def uneven_conf():
    """Layers that share no size, odd widths everywhere, every kind of feed-forward behind every mixer and none."""
    return conf([latent(3, 20, 6, 12, 36, 0.3, experts(5, 2, 20, 28)), retention(3, 12, 20, None),
                 latent(2, 10, 14, 30, 50, 0.2, dense(36), base=90.0, factor=1.5, original=200, fast=30.0, slow=1.0),
                 retention(1, 40, 70, experts(9, 3, 12, 44), decay=[0.93]), latent(5, 8, 4, 8, 24, 0.4, None),
                 retention(2, 24, 6, dense(52), decay=[0.5, 1.0])], width=44, vocab=75)


def round_conf():
    """Sizes the tensor-core kernels take without padding."""
    return conf([retention(4, 64, 128, dense(384)), latent(8, 64, 32, 64, 128, 0.11, experts(16, 4, 128, 128), original=300),
                 retention(2, 128, 64, experts(7, 1, 64, 256)), latent(4, 128, 64, 128, 256, 0.08, dense(256), base=9000.0)],
                width=256, vocab=320)

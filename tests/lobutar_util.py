"""Small Lobutar configurations for the tests."""
import torch

from tests import plan_util
from tests.oracle import lobutar as oracle
from tests.plan_util import make_engine, make_rows, rms_error, run_alone, run_mixed, tokens  # noqa: F401


def rotation(dims, base):
    return dict(dims=dims, base=base)


def attention(heads, kv_heads, dim, vdim, rot, scale, diff, mlp, base=400.0):
    return dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff,
                                                      rot=rotation(rot, base)))


def latent(heads, dim, rot_dim, vdim, kv_rank, window, scale, mlp, base=600.0):
    return dict(type="latent_attention", mlp=mlp, mixer=dict(
        heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, mask=dict(size=window),
        rot=rotation(rot_dim, base)))


def again(layers, j):
    """A layer that runs layer j's weights once more."""
    return dict(type=layers[j]["type"], mixer=layers[j]["mixer"], mlp=layers[j]["mlp"], weights_of=j)


def dense(ff):
    return dict(kind="dense", ff=ff)


def experts(n, top, ff, shared, groups=1, keep=1, scale=1.0):
    return dict(kind="moe", expert=dict(ff=ff), shared=dict(ff=shared) if shared else None,
                router=dict(experts=n, top=top, scale=scale, groups=dict(count=groups, keep=keep)))


def conf(layers, width, vocab, streams=2, eps=1e-5):
    return dict(architecture="Lobutar", layers=layers, norm=dict(eps=eps), streams=streams, vocab=vocab, width=width)


def uneven_conf():
    """Layers that share no size, odd widths everywhere, every kind of feed-forward behind every mixer and none, a layer that
    comes back twice with others between."""
    ly = [attention(6, 2, 20, 12, 6, 0.3, 0.2, experts(6, 2, 20, 28, groups=3, keep=2, scale=2.5)),
          latent(3, 20, 6, 12, 36, 9, 0.3, dense(36)),
          attention(3, 3, 10, 30, 10, 0.25, 0.55, None, base=90.0),
          latent(2, 10, 14, 30, 50, 1, 0.2, experts(5, 3, 12, 0), base=50.0)]
    ly.append(again(ly, 0))
    ly += [attention(1, 1, 12, 4, 2, 0.4, 0.0, dense(52)), latent(5, 8, 4, 8, 24, 70, 0.4, None), again(ly, 0)]
    ly.append(again(ly, 6))
    return conf(ly, width=44, vocab=75, streams=3)


def round_conf():
    """Sizes the tensor-core kernels take without padding."""
    ly = [attention(8, 2, 64, 128, 64, 0.11, 0.4, dense(384)),
          latent(8, 64, 32, 64, 128, 48, 0.11, experts(16, 4, 128, 128, groups=4, keep=2, scale=1.7)),
          attention(4, 4, 128, 64, 32, 0.08, 0.7, experts(12, 3, 64, 256, groups=2, keep=1, scale=0.8), base=9000.0)]
    ly += [again(ly, 1), latent(4, 128, 64, 128, 256, 100, 0.08, dense(256), base=9000.0), again(ly, 2)]
    return conf(ly, width=256, vocab=320, streams=2)


def decisive(W, c, level=4.0):
    """The same weights with expert choices that bf16 rounding cannot turn: the residual's first column carries the token's
    parity untouched through every layer, the routers read mainly that, and the corrections are well apart."""
    W = dict(W)
    W["embed"] = W["embed"].clone()
    W["embed"][:, 0] = torch.tensor([level, -level]).repeat(c["vocab"])[:c["vocab"]]
    for k, v in W.items():
        end = k.rsplit(".", 1)[-1]
        if end == "down" or k.endswith((".mix.o", ".mix.o.b")):
            W[k] = v.clone()
            W[k][0] = 0
        elif end in ("norm1", "norm2"):
            W[k] = v.clone()
            W[k][0] = 1
        elif end in ("in", "mix") and ".hc" in k:       # the streams' parities add up and keep their size
            W[k] = (v.abs().float() / v.abs().float().sum(0)).to(v.dtype)
        elif end == "router":
            E = v.shape[0]
            W[k] = v * 0.1
            W[k][:, 0] = torch.tensor([1.0, -1.0, 1.0, 1.0, -1.0, -1.0, -1.0]).repeat(E)[:E]
        elif end == "correction":
            E = v.shape[0]
            W[k] = (torch.arange(E) * 5 % 17 * 0.3 / 17 + torch.arange(E) * 0.7 / E).to(v.dtype)
    return W


def weights(c, seed, dtype="float32"):
    """Random weights, for bf16 with expert choices that rounding cannot turn."""
    W = oracle.random_weights(c, seed=seed)
    return decisive(W, c) if dtype == "bfloat16" else W


def assert_close(got, want, dtype="float32", what=None):
    if dtype == "float32":
        return plan_util.assert_close(got, want, dtype, what)
    e = rms_error(got, want)
    assert e.max() < 0.1 and e.quantile(0.9) < 0.03, (what, float(e.max()), float(e.quantile(0.9)), int(e.argmax()))

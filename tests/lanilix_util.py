"""Small Lanilix configurations; the driver and the error measures are those of the other mixer stacks (ludesun_util)."""
import lanilix_oracle as oracle
from ludesun_util import check, cut, err, feed, make_engine, seq   # noqa: F401

DELTA_ODD = dict(heads=3, kv_heads=1, dim=7, vdim=10, conv=3)
DELTA_EVEN = dict(heads=4, kv_heads=2, dim=24, vdim=40, conv=4)
DELTA_ONE = dict(heads=1, kv_heads=1, dim=1, vdim=1, conv=1)


def attn(heads, kv_heads, dim, window, keep, rot, base=1000.0, scale=None):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale or dim ** -0.5, mask=dict(size=window, keep_first=keep),
                rot=dict(base=base, dims=rot))


ATTN_ODD = attn(6, 2, 10, 9, 3, 6)
ATTN_EVEN = attn(4, 4, 24, 21, 0, 24, 50.0, 0.3)
ATTN_ONE = attn(1, 1, 2, 1, 1, 2, 10.0, 1.0)


def layer(kind, mixer, ff=None, limit=1.5, **kw):
    return dict(type=kind, mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff, limit=limit), **kw)


def model(width, vocab, *layers, eps=1e-5):
    return dict(architecture="Lanilix", vocab=vocab, width=width, norm=dict(eps=eps), layers=list(layers))


ODD = model(37, 61, layer("delta", DELTA_ODD, 45), layer("attention", ATTN_ODD), layer("delta", DELTA_ODD, 51, 0.7),
            layer("attention", ATTN_ODD, weights_of=1), layer("delta", DELTA_ODD, 45, weights_of=0), eps=3e-5)
EVEN = model(64, 88, layer("attention", ATTN_EVEN, 128, 0.4), layer("delta", DELTA_EVEN, 72), layer("delta", DELTA_EVEN),
             layer("delta", DELTA_EVEN, 72, weights_of=1))
ONE = model(8, 17, layer("delta", DELTA_ONE, 8), layer("attention", ATTN_ONE, 1), layer("delta", DELTA_ONE))
CONFIGS = {"odd": ODD, "even": EVEN, "one": ONE}


def reference(cfg, sd, toks):
    return {k: oracle.forward(cfg, sd, t) for k, t in toks.items()}

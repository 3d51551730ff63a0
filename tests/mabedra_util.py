"""Small Mabedra configurations; the driver and the error measures are those of the other mixer stacks (ludesun_util)."""
import mabedra_oracle as oracle
from ludesun_util import check, cut, err, feed, make_engine, seq   # noqa: F401


def attn(heads, kv_heads, dim, vdim, window, rot, base=1000.0, scale=None, diff=0.4, scaling=(8.0, 1.0, 4.0, 256)):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, diff=diff, mask=dict(size=window),
                rot=dict(base=base, dims=rot, scaling=dict(zip(("factor", "low", "high", "original"), scaling))))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, shared=None):
    out = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    return dict(out, shared=dict(ff=shared)) if shared else out


def layer(mixer, mlp=None):
    return dict(type="attention", mixer=mixer, mlp=mlp)


def model(width, vocab, *layers, eps=1e-5, taps=4):
    return dict(architecture="Mabedra", vocab=vocab, width=width, canon=dict(taps=taps), norm=dict(eps=eps), layers=list(layers))


A_ODD = attn(3, 1, 10, 14, 9, 6)
A_EVEN = attn(8, 2, 24, 40, 21, 24, 50.0, 0.3, 0.7, (3.0, 0.5, 6.0, 64))
A_ONE = attn(1, 1, 2, 1, 1, 2, 10.0, 1.0, 0.1)
ODD = model(37, 61, layer(A_ODD, moe(5, 3, 11, 9)), layer(A_ODD), layer(attn(6, 2, 9, 5, 20, 4), dense(45)), layer(A_ODD, moe(7, 1, 13)), eps=3e-5, taps=5)
EVEN = model(64, 88, layer(A_EVEN, dense(96)), layer(A_EVEN, moe(6, 2, 48, 72)), layer(attn(4, 4, 32, 64, 17, 16), moe(3, 3, 128, 128)), layer(A_EVEN), taps=2)
ONE = model(8, 17, layer(A_ONE, dense(1)), layer(A_ONE, moe(1, 1, 1, 1)), taps=1)
CONFIGS = {"odd": ODD, "even": EVEN, "one": ONE}


def reference(cfg, sd, toks):
    return {k: oracle.forward(cfg, sd, t) for k, t in toks.items()}

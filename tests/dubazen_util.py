"""Small Dubazen configurations; the driver and the error measures are those of the other mixer stacks (ludesun_util)."""
import dubazen_oracle as oracle
from ludesun_util import check, cut, err, feed, make_engine, seq   # noqa: F401


def turn(heads, kv_heads, dim, vdim, rot, base=1000.0, scale=None):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, rot=dict(base=base, dims=rot))


def decay(heads, dim, vdim, rates):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=list(rates))


def pair(left, right, a=0.7, b=1.3):
    return dict(type="parallel", mixer=dict(left=left, right=right, left_scale=a, right_scale=b))


def gla(heads, dim, vdim, tau):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau))


def mamba(inner, state, rank, conv):
    return dict(type="mamba1", mixer=dict(inner=inner, state=state, dt_rank=rank, conv=conv))


def moe(experts, top, ff, shared, limit=1.5, shared_limit=0.8):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top), shared=dict(ff=shared, limit=shared_limit))


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def model(width, vocab, *layers, eps=1e-5, streams=3, scale=2.0):
    return dict(architecture="Dubazen", vocab=vocab, width=width, streams=streams, embedding=dict(scale=scale), norm=dict(eps=eps), layers=list(layers))


P_ODD = pair(turn(3, 1, 10, 14, 6), decay(2, 7, 9, (0.6, 0.97)))
P_EVEN = pair(turn(8, 2, 40, 32, 24, 50.0, 0.4), decay(4, 32, 48, (0.5, 0.9, 0.99, 0.999)), 1.2, -0.6)
P_ONE = pair(turn(1, 1, 1, 2, 0, 10.0, 1.0), decay(1, 1, 1, (1.0,)))
ODD = model(37, 61, layer(P_ODD, moe(5, 3, 11, 9)), layer(gla(3, 6, 5, 3.0)), layer(mamba(21, 5, 3, 5), moe(7, 1, 13, 4)), layer(P_ODD), eps=3e-5, streams=5, scale=3.0)
EVEN = model(64, 88, layer(mamba(96, 16, 8, 4), moe(6, 2, 48, 72)), layer(gla(4, 24, 32, 10.0), moe(3, 3, 128, 128)), layer(P_EVEN, moe(6, 2, 48, 72)),
             layer(gla(2, 64, 16, 1.0)), streams=4)
ONE = model(8, 17, layer(P_ONE, moe(1, 1, 1, 1)), layer(gla(1, 1, 1, 1.0), moe(1, 1, 1, 1)), layer(mamba(1, 1, 1, 1)), streams=1, scale=1.0)
CONFIGS = {"odd": ODD, "even": EVEN, "one": ONE}


def reference(cfg, sd, toks):
    return {k: oracle.forward(cfg, sd, t) for k, t in toks.items()}

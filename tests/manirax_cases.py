"""Small configurations of the Manirax design for the tests: sizes of their own, every branch of the design somewhere."""
from __future__ import annotations


def layer(heads=4, kv_heads=2, dim=32, vdim=32, scale=0.2, rot=(16, 10000.0, 4.0), r_heads=3, r_dim=24, r_vdim=40,
          decay=(0.5, 0.9, 0.995), left_scale=0.7, right_scale=1.3, ff=80) -> dict:
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if rot is not None:
        left["rot"] = dict(dims=rot[0], base=rot[1], **({} if rot[2] is None else dict(scaling=dict(factor=rot[2]))))
    return dict(type="parallel", mlp=None if ff is None else dict(kind="dense", ff=ff),
                mixer=dict(left=left, left_scale=left_scale, right_scale=right_scale,
                           right=dict(heads=r_heads, dim=r_dim, vdim=r_vdim, decay=list(decay))))


def config(layers, vocab=331, width=72, eps=1e-5, alpha=1.7) -> dict:
    return dict(architecture="Manirax", vocab=vocab, width=width, norm=dict(eps=eps), postln_alpha=alpha, layers=layers)


CONFIGS = {
    # head sizes equal and unequal, grouped and not, layers of different sizes, one without a feed-forward
    "mixed": config([
        layer(),
        layer(heads=6, kv_heads=1, dim=64, vdim=48, rot=(64, 5000.0, 1.0), r_heads=2, r_dim=64, r_vdim=64, decay=(0.8, 0.99), ff=None),
        layer(heads=3, kv_heads=3, dim=80, vdim=96, scale=0.05, rot=(20, 300.0, 7.5), r_heads=1, r_dim=33, r_vdim=17, decay=(0.97,)),
    ]),
    # sizes no vector width divides, no rotation, a decay of one and one of zero, scales of one
    "odd": config([
        layer(heads=5, kv_heads=5, dim=21, vdim=19, rot=None, r_heads=2, r_dim=13, r_vdim=11, decay=(1.0, 0.0), ff=37, left_scale=1.0, right_scale=1.0),
        layer(heads=2, kv_heads=1, dim=10, vdim=7, rot=(10, 77.0, None), r_heads=4, r_dim=8, r_vdim=8, decay=(0.1, 0.6, 0.9, 0.999), ff=50),
    ], vocab=97, width=45, eps=1e-3, alpha=1.0),
    # tensor-core sizes: 64 and 128 channels, more than eight and more than sixteen query heads per key head
    "wide": config([
        layer(heads=24, kv_heads=1, dim=64, vdim=128, scale=0.1, rot=(32, 1e5, 2.0), r_heads=2, r_dim=128, r_vdim=64, decay=(0.7, 0.998), ff=256),
        layer(heads=12, kv_heads=1, dim=128, vdim=64, scale=0.06, rot=(128, 1e4, 8.0), r_heads=4, r_dim=64, r_vdim=128, decay=(0.3, 0.9, 0.99, 0.9995), ff=192),
    ], vocab=512, width=256, alpha=2.5),
    # one head size throughout, a second wide layer whose keys and values are 128 channels
    "even": config([
        layer(heads=6, kv_heads=2, dim=64, vdim=64, scale=0.11, rot=(48, 2e4, 2.5), r_heads=3, r_dim=64, r_vdim=64, decay=(0.5, 0.93, 0.998), ff=136),
        layer(heads=3, kv_heads=1, dim=128, vdim=128, scale=0.07, rot=(128, 1e6, 1.5), r_heads=2, r_dim=128, r_vdim=128, decay=(0.85, 0.9999), ff=104),
    ], vocab=264, width=136, alpha=2.0),
    # more channels per head than the tensor-core forms take
    "large_heads": config([layer(heads=2, kv_heads=1, dim=160, vdim=144, rot=(96, 1e4, 3.0), r_heads=1, r_dim=136, r_vdim=130, decay=(0.95,))]),
}

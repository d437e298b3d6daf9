"""Small configurations of the Gotunex design for the tests: sizes of their own, every branch of the design somewhere."""
from __future__ import annotations


def latent(heads=3, dim=24, rot_dim=16, vdim=20, q_rank=36, kv_rank=56, scale=0.17, base=10000.0, kv_from=None, mlp=None) -> dict:
    mixer = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dim))
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=mixer, mlp=mlp)


def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, mlp=None) -> dict:
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=mlp)


def dense(ff=96) -> dict:
    return dict(kind="dense", ff=ff)


def moe(experts=7, top=3, ff=40) -> dict:
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))


def config(layers, vocab=331, width=88, eps=1e-5, scale=3.5) -> dict:
    return dict(architecture="Gotunex", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)


CONFIGS = {
    # both mixers under every kind of feed-forward, a cache read by two later layers that differ from its owner, two delta layers apart
    "mixed": config([
        delta(mlp=moe()),
        latent(mlp=dense()),
        latent(heads=5, dim=32, vdim=12, q_rank=28, scale=0.3, kv_from=1, mlp=moe(experts=3, top=1, ff=72)),
        latent(heads=2, kv_rank=72, rot_dim=32, base=500.0, mlp=None),
        delta(heads=3, kv_heads=3, dim=16, vdim=16, conv=3, mlp=dense(60)),
        latent(heads=4, dim=8, vdim=36, kv_from=1, mlp=moe(experts=12, top=4, ff=24)),
    ]),
    # sizes no vector width divides, one head, one tap, every expert chosen, scale one
    "odd": config([
        latent(heads=1, dim=7, rot_dim=6, vdim=5, q_rank=11, kv_rank=13, base=77.0, scale=1.0, mlp=moe(experts=2, top=2, ff=9)),
        delta(heads=3, kv_heads=1, dim=10, vdim=7, conv=1, mlp=dense(37)),
        latent(heads=3, dim=9, rot_dim=6, vdim=11, q_rank=17, kv_rank=13, base=77.0, kv_from=0, mlp=None),
        delta(heads=2, kv_heads=2, dim=13, vdim=21, conv=6, mlp=None),
    ], vocab=97, width=45, eps=1e-3, scale=1.0),
    # sizes of the tensor-core forms, more heads than one block holds
    "wide": config([
        latent(heads=20, dim=64, rot_dim=32, vdim=64, q_rank=128, kv_rank=256, scale=0.1, mlp=moe(experts=16, top=2, ff=192)),
        delta(heads=4, kv_heads=2, dim=64, vdim=64, mlp=dense(320)),
        latent(heads=36, dim=48, rot_dim=32, vdim=80, q_rank=96, kv_rank=256, scale=0.11, kv_from=0, mlp=moe(experts=5, top=2, ff=136)),
    ], vocab=520, width=256, scale=16.0),
    # the largest latents and heads
    "deep": config([
        delta(heads=2, kv_heads=1, dim=128, vdim=128, conv=4, mlp=moe(experts=6, top=1, ff=130)),
        latent(heads=6, dim=128, rot_dim=64, vdim=128, q_rank=192, kv_rank=512, scale=0.07, base=1e6, mlp=dense(200)),
        latent(heads=3, dim=100, rot_dim=64, vdim=96, q_rank=64, kv_rank=320, scale=0.09, mlp=None),
    ], vocab=264, width=200, scale=9.0),
    # more channels than the tensor-core forms take
    "large_heads": config([
        latent(heads=2, dim=140, rot_dim=96, vdim=150, q_rank=60, kv_rank=600, scale=0.06, mlp=dense(50)),
        delta(heads=2, kv_heads=1, dim=160, vdim=144, conv=2, mlp=None),
    ]),
}

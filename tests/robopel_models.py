"""Small configurations of the Robopel design for tests: every branch, and sizes that are odd, equal, one,
or larger than a tensor-core tile."""
import robopel_plain as P

A, G, C = P.attention, P.mingru, P.make_config
MODELS = {
    # two readers of one cache with other windows, blocks, caps and numbers of query heads
    "shared": C(layers=[A(mlp=P.moe(5, 1, 2, 40)), G(56, P.dense(72)), A(size=33, pool=4, scale=0.4, softcap=25.0, kv_from=0),
                        G(40, P.moe(6, 2, 3, 24)), A(size=11, pool=6, scale=0.5, softcap=None, kv_from=0, mlp=P.dense(33))]),
    # nothing is a multiple of anything; no caps, plain rotation of a part of the head
    "odd": C(width=50, vocab=77, eps=1e-4, layers=[A(heads=3, kv_heads=1, dim=10, vdim=9, size=7, pool=3, turn=P.rot(4, 30.0, None), softcap=None,
                                                     mlp=P.dense(21)), G(37), A(heads=1, kv_heads=1, dim=7, vdim=13, size=16, pool=5,
                                                                                turn=P.rot(6, 500.0), mlp=P.moe(3, 2, 2, 15))]),
    # more query heads per key head than a tensor-core tile has rows; blocks of one token; every expert chosen
    "many": C(width=72, vocab=130, embed_scale=1.0, layers=[A(heads=20, kv_heads=1, dim=16, vdim=16, size=40, pool=1, mlp=P.moe(3, 0, 3, 48)),
                                                            A(heads=34, kv_heads=2, dim=24, vdim=8, size=25, pool=40, turn=P.rot(8))]),
    # tensor-core sizes
    "wide": C(width=128, vocab=320, eps=1e-3, embed_scale=0.7,
              layers=[G(256, P.moe(9, 3, 4, 128)), A(heads=8, kv_heads=2, dim=32, vdim=64, size=48, pool=16, turn=P.rot(32, 1e4, (4.0, 1.0, 2.0, 4000)),
                                                     softcap=50.0, mlp=P.dense(512)), A(heads=4, kv_heads=2, dim=32, vdim=64, size=70, pool=8,
                                                                                        turn=P.rot(32), kv_from=1, mlp=P.moe(4, 1, 1, 72))]),
    # a window of one token, blocks alone; a window without blocks; everything visible; no rotation
    "edges": C(width=40, vocab=90, layers=[A(heads=4, kv_heads=1, dim=24, vdim=24, size=1, pool=5, turn=None, mlp=P.dense(64)),
                                           A(heads=4, kv_heads=4, dim=8, vdim=8, size=9, pool=None, turn=P.rot(8), mlp=P.moe(6, 2, 3, 16)),
                                           A(heads=2, kv_heads=2, dim=16, vdim=16, size=1000, pool=7, mlp=None), G(24)]),
}


def weights(name):
    return P.make_weights(MODELS[name], sum(map(ord, name)))

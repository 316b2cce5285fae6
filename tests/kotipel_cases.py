"""Small random models of the Kotipel design for the tests: sizes that are no multiples of tiles, equal and single head
counts, groups that do not end at heads, loops of every shape, layers without a feed-forward, models without a token
input, and sizes that the tensor-core kernels take. Queries are scaled up so that single keys dominate, and decays are
slow for some channels, so that a lost key or state shows in the output."""

from flashrec_b200.kotipel import KotipelConfig, random_tensors


def par(heads, kv, dim, vdim, rot, gla, tau=16.0, scaling=(8.0, 1.0, 4.0, 64), base=5000.0, scale=None, ff=72, limit=0.8):
    r = dict(dims=rot, base=base)
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return dict(type="parallel", mlp=None if ff is None else dict(kind="dense", ff=ff, limit=limit), mixer=dict(
        left=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rot=r, scale=scale or dim ** -0.5),
        right=dict(heads=gla[0], dim=gla[1], vdim=gla[2], tau=tau)))


def mamba(heads, vdim, state, groups, conv, norm_groups, ff=72, limit=0.8):
    return dict(type="mamba2", mlp=None if ff is None else dict(kind="dense", ff=ff, limit=limit), mixer=dict(
        heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups))


def config(vocab, width, layers, loop=None, side=None, eps=1e-5):
    cfg = dict(architecture="Kotipel", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side:
        cfg["token_side"] = dict(dim=side)
    return cfg


CASES = {
    # nothing a multiple of 16; three query heads per kv head; norm parts that cut through heads; a loop over both kinds
    "ragged": config(131, 90, [mamba(6, 10, 12, 2, 3, 4), par(6, 2, 20, 24, 12, (3, 18, 22)), mamba(3, 20, 9, 3, 5, 1, ff=None),
                               par(6, 3, 24, 12, 24, (5, 7, 11), tau=3.0, scaling=None)], loop=(0, 2, 3), side=11),
    # heads == kv heads, no scaling, one layer run three times at the end, sizes of whole tiles
    "equal": config(200, 128, [mamba(4, 32, 32, 4, 4, 4, ff=160), par(2, 2, 64, 64, 64, (2, 64, 32), scaling=None, ff=160)],
                    loop=(1, 2, 3), side=32, eps=1e-3),
    # one kv head, wide heads, no token input, no loop; the decays as they come (tau 1)
    "single_kv": config(97, 160, [par(4, 1, 128, 128, 32, (2, 64, 64), tau=1.0, ff=200), mamba(2, 64, 64, 1, 2, 2, ff=64)]),
    # one head everywhere, one tap, a loop over everything run once
    "one_head": config(67, 64, [par(1, 1, 32, 48, 16, (1, 16, 16), ff=None), mamba(1, 16, 16, 1, 1, 1, ff=40),
                                par(1, 1, 16, 16, 2, (1, 40, 96), ff=33)], loop=(0, 3, 1), side=8),
    # the shapes of real layers on the tensor cores: long state, several heads per group, wide values
    "tiles": config(160, 192, [mamba(8, 64, 128, 2, 4, 2, ff=128), par(4, 2, 64, 128, 32, (3, 128, 128), ff=128),
                               mamba(4, 128, 64, 1, 4, 1, ff=None)], side=24),
    # only recurrences: no cache at all
    "recurrent": config(80, 48, [mamba(3, 16, 8, 1, 4, 3, ff=32), mamba(2, 24, 40, 2, 2, 1, ff=None)], loop=(1, 2, 2), side=5),
}


def make(name, seed=1, sharp=2.5):
    """(config dict, parsed config, bf16 tensors)"""
    raw = CASES[name]
    cfg = KotipelConfig.from_json(raw)
    tensors = random_tensors(cfg, seed, rank=5 if name == "ragged" else 16)
    for k, t in tensors.items():
        if k.endswith("left.q.norm"):
            tensors[k] = (t.float() * sharp).to(t.dtype)
        if k.endswith("a2.b"):  # every third channel keeps its state for long
            t = t.float()
            t[::3] += 4
            tensors[k] = t.to(tensors[k].dtype)
        if k == "loop.step":
            tensors[k] = (t.float() * 8).to(t.dtype)
    return raw, cfg, tensors


def tokens(cfg, n, seed=0):
    import torch

    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg.vocab, (n,), generator=g).tolist()

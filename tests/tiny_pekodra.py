"""Tiny Pekodra configurations of the tests' own, and a folder of random weights shaped so that faults show.

Sizes differ from layer to layer and between the configurations: query heads over 1, 2 or as many key/value heads,
value heads smaller and larger than the keys', rotations of a whole head, of a part and of nothing, with and without
a blend of the rates (edges inside and outside the pairs), windows of one token, of less and of more than a page, and
longer than the prompts; dense and routed feed-forwards and none, one and several experts a token, with and without the
expert that every token passes, of another size than the routed ones; loops over one layer, over all layers, once and
three times, and no loop; widths that are no multiple of 8; scales, eps and multipliers of their own.
"""

import json
from pathlib import Path

import torch

BLEND = dict(factor=6.0, original=48, fast=8.0, slow=0.5)  # its edges lie inside the pairs of a part of 16 at base 300


def attn(heads, kv_heads, dim, vdim, window, scale, base, dims, scaling=None):
    rot = dict(base=base, dims=dims)
    if scaling is not None:
        rot["scaling"] = scaling
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window), rot=rot, scale=scale)


ATT = attn(6, 2, 24, 16, 21, 0.5, 300.0, 16, BLEND)
ATT_FULL = attn(4, 4, 16, 24, 50, 0.6, 10000.0, 16, dict(factor=2.5, original=300, fast=4.0, slow=1.0))
ATT_ODD = attn(3, 1, 20, 28, 33, 0.45, 1000000.0, 6, dict(factor=1.5, original=1000, fast=32.0, slow=1.0))
ATT_SELF = attn(5, 5, 12, 10, 1, 0.7, 500.0, 4)     # every position sees itself only
ATT_BARE = attn(12, 2, 8, 8, 1000, 0.9, 100.0, 0)  # no rotation; a window longer than any prompt here
ATT_MID = attn(8, 2, 64, 48, 90, 0.2, 10000.0, 32, dict(factor=8.0, original=512, fast=16.0, slow=2.0))
# values of the keys' size, at sizes that the kernels for plain attention take
ATT_EVEN = attn(6, 2, 16, 16, 27, 0.6, 10000.0, 12, dict(factor=2.0, original=200, fast=8.0, slow=1.0))
ATT_EVEN32 = attn(4, 1, 32, 32, 40, 0.3, 300.0, 32, BLEND)
ATT_EVEN64 = attn(8, 2, 64, 64, 75, 0.2, 10000.0, 32, dict(factor=8.0, original=512, fast=16.0, slow=2.0))
ATT_EVEN128 = attn(2, 2, 128, 128, 66, 0.1, 500000.0, 128, dict(factor=5.0, original=300, fast=16.0, slow=1.0))
ATT_MID2 = attn(4, 4, 32, 64, 64, 0.35, 500000.0, 32, dict(factor=3.0, original=128, fast=32.0, slow=1.0))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, shared=None):
    out = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared is not None:
        out["shared"] = dict(ff=shared)
    return out


def layer(mixer, mlp):
    return dict(type="attention", mixer=json.loads(json.dumps(mixer)), mlp=mlp)


def model(width, vocab, layers, loop=None, eps=1e-5, logit_scale=0.7, embedding_scale=3.0):
    out = dict(architecture="Pekodra", width=width, vocab=vocab, norm=dict(eps=eps), layers=layers, logit_scale=logit_scale,
               embedding=dict(scale=embedding_scale))
    if loop is not None:
        out["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return out


CONFIGS = {
    "mix": model(80, 200, [
        layer(ATT, moe(24, 6, 2, shared=40)),
        layer(ATT_FULL, dense(48)),
        layer(ATT_SELF, moe(16, 5, 1, shared=16)),
        layer(ATT_BARE, None),
        layer(ATT, dense(24)),
    ], loop=(1, 4, 3)),
    "odd": model(52, 90, [layer(ATT_ODD, moe(20, 4, 2, shared=12)), layer(ATT_BARE, dense(36)), layer(ATT_FULL, None),
                          layer(ATT_SELF, moe(12, 7, 3))],
                 loop=(0, 4, 2), eps=1e-6, logit_scale=1.3, embedding_scale=0.25),
    # sizes that are multiples of nothing much: rows of 50 and 77; a loop of one pass
    "ragged": model(50, 77, [layer(ATT_BARE, moe(10, 3, 2, shared=6)), layer(ATT_ODD, dense(14)), layer(ATT_SELF, None)], loop=(1, 2, 1),
                    eps=1e-3, logit_scale=-2.2, embedding_scale=1.0),
    "alone": model(48, 120, [layer(ATT, dense(24)), layer(ATT_ODD, moe(24, 4, 1, shared=24))], embedding_scale=11.5),  # no loop at all
    "even": model(64, 110, [layer(ATT_EVEN, dense(32)), layer(ATT_EVEN64, moe(32, 4, 2, shared=24)), layer(ATT_EVEN128, None),
                            layer(ATT_EVEN32, dense(48))], loop=(1, 3, 2), embedding_scale=1.5),
    # sizes that the tensor-core kernels take, with a looped last layer
    "mid": model(128, 300, [layer(ATT_MID, dense(192)), layer(ATT_MID2, moe(64, 8, 2, shared=64)), layer(ATT_MID, moe(136, 4, 1, shared=192))],
                 loop=(2, 3, 2), eps=1e-6, logit_scale=0.5, embedding_scale=2.0),
}
PAGE = {"mix": 8, "odd": 16, "ragged": 32, "alone": 64, "even": 64, "mid": 64}
LENGTHS = {"mix": [1, 45, 2, 97, 33, 130, 64], "odd": [70, 3, 41, 100], "ragged": [75, 2, 140], "alone": [90, 1, 150],
           "even": [150, 40, 2, 210], "mid": [200, 129, 64]}
LOUD = 1.0  # how far the directions that the routers read stand out of the rest of an embedding
TOL = {"float32": 3e-5, "bfloat16": 2e-2}  # largest |difference| over largest |reference logit|


def make_folder(config, seed, folder, std=0.08):
    """A model folder with random weights of deviation ``std`` (a wide model wants a smaller one), biases and norm
    weights that are not small, a joining matrix that lets both the stream and the embedding's output through, and
    routing that is rarely a close call: the embeddings hold a handful of orthogonal directions in an order of their own
    per token, with sizes that are well apart, and every router's rows point along them (undoing its norm's weights)."""
    from safetensors.torch import save_file

    from akas_b200.config import config_from_dict
    from akas_b200.weights import random_tensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    tensors = random_tensors(config_from_dict(config), seed=seed, std=std, dtype="float32")
    g = torch.Generator().manual_seed(seed + 1)
    c = config["width"]
    for name in list(tensors):
        if name.endswith(("norm1", "norm2", "final.norm")):
            tensors[name] = torch.randn(tensors[name].shape, generator=g) * 0.3
        if name.endswith(".b"):
            tensors[name] = torch.randn(tensors[name].shape, generator=g) * 0.3
        if name == "loop.in":
            noise = torch.randn(tensors[name].shape, generator=g) * (0.3 / c ** 0.5)
            tensors[name] = torch.cat([0.7 * torch.eye(c), 0.6 * torch.eye(c)], dim=1) + noise
    most = max([entry["mlp"]["router"]["experts"] for entry in config["layers"] if entry["mlp"] and entry["mlp"]["kind"] == "moe"] + [1])
    directions = torch.linalg.qr(torch.randn(c, most, generator=g))[0].T
    sizes = torch.linspace(-1.0, 1.0, most) if most > 1 else torch.ones(1)
    orders = torch.stack([sizes[torch.randperm(most, generator=g)] for _ in range(config["vocab"])])
    apart = LOUD * c ** 0.5 * (3.0 / most) ** 0.5
    tensors["embed"] = (torch.randn(tensors["embed"].shape, generator=g) + apart * orders @ directions) / config["embedding"]["scale"]
    for name in list(tensors):
        if name.endswith("mlp.router"):
            experts = tensors[name].shape[0]
            rows = directions[torch.randperm(most, generator=g)[:experts]]
            tensors[name] = rows * (most / c ** 0.5) / (1.0 + tensors[name.replace("mlp.router", "norm2")])
    tensors = {k: v.to(torch.bfloat16).contiguous() for k, v in tensors.items()}  # stored as a checkpoint stores them
    save_file(tensors, str(folder / "model.safetensors"))
    (folder / "config.json").write_text(json.dumps(config))
    return folder, {k: v.to(torch.float64) for k, v in tensors.items()}


def plant(folder, config, key_token, query_token, strength=0.7):
    """Rewrites a folder so that in layer 0 ``query_token``'s queries and ``key_token``'s keys are long along one channel
    that the rotation leaves alone: wherever the two stand, the query's score for that key is far above the others', so
    the key is felt among hundreds. The two tokens' embeddings are two orthogonal vectors of +-1 (layer 0's first norm
    weighs all channels alike here); the channel's row of every query head points along the query token's, of every key
    head along the key token's. The joining matrix, if there is one, passes both its halves."""
    from safetensors.torch import load_file, save_file

    m = config["layers"][0]["mixer"]
    channel, c = m["dim"] - 1, config["width"]
    assert m["rot"]["dims"] <= channel
    u, u2 = torch.ones(c), torch.ones(c)
    u[1::2] = -1.0
    u2[2::4] = u2[3::4] = -1.0
    path = str(Path(folder) / "model.safetensors")
    t = load_file(path)
    t["embed"][key_token], t["embed"][query_token] = u.to(torch.bfloat16), u2.to(torch.bfloat16)
    t["l0.norm1"] = torch.zeros_like(t["l0.norm1"])
    for a in range(m["heads"]):
        t["l0.mix.q"][a * m["dim"] + channel] = (strength * u2 / c ** 0.5).to(torch.bfloat16)
    for a in range(m["kv_heads"]):
        t["l0.mix.k"][a * m["dim"] + channel] = (strength * u / c ** 0.5).to(torch.bfloat16)
    t["l0.mix.v"] = (t["l0.mix.v"].float() * 4.0).to(torch.bfloat16)
    if "loop.in" in t:
        t["loop.in"] = torch.cat([0.5 * torch.eye(c), 0.5 * torch.eye(c)], dim=1).to(torch.bfloat16)
    save_file(t, path)
    return {k: v.to(torch.float64) for k, v in t.items()}


def prompts(vocab, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lengths]

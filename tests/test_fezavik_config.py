"""The Fezavik configuration, its model spec, the tensors it declares, and what the cache manager is asked for (keys and
values for a window in attention layers, one latent row per token in latent layers, a state slot in recurrent ones); the
stretched frequencies; the block between two norms in plain operations; no GPU."""
import copy

import pytest
import torch

from helpers import TINY_FEZAVIK, make_fezavik_folder
from plain import fezavik_plain as plain
from photon_infer_b200.cache.manager import CacheManager
from photon_infer_b200.config import get_architecture, load_config
from photon_infer_b200.config.fezavik_config import FezavikConfig
from photon_infer_b200.errors import ErrorCode, PhotonError
from photon_infer_b200.models.model import _Skeleton, declared_tensors
from photon_infer_b200.parts.base import FeedForward, Mixer, Norm, Normed, PagedCacheSpec
from photon_infer_b200.parts.block import SandwichBlock
from photon_infer_b200.parts.registry import create_part
from photon_infer_b200.parts.rope import scaled_frequencies


def _cfg(name):
    return copy.deepcopy(TINY_FEZAVIK[name]["config"])


def load_spec(name_or_dict):
    arch = get_architecture("Fezavik")
    return arch.build_spec(arch.config_class.from_dict(_cfg(name_or_dict) if isinstance(name_or_dict, str) else name_or_dict))


def test_round_trip_and_registry(tmp_path):
    for name in TINY_FEZAVIK:
        cfg = FezavikConfig.from_dict(_cfg(name))
        assert FezavikConfig.from_dict(cfg.to_dict()) == cfg
    arch, cfg = load_config(make_fezavik_folder(str(tmp_path / "m"), "fv_a"))
    assert arch.name == "Fezavik" and cfg.width == 64 and [l.type for l in cfg.layers] == ["attention", "hgrn2", "latent_attention", "attention"]
    d = _cfg("fv_b"); d["architectures"] = [d.pop("architecture")]
    assert FezavikConfig.from_dict(d).architecture == "Fezavik"


@pytest.mark.parametrize("path,value,word", [
    (("width",), None, "width"), (("vocab",), 0, "vocab"), (("norm", "eps"), None, "norm.eps"), (("norm",), None, "norm"),
    (("layers", 1, "type"), "gla", "layers[1].type"), (("layers", 1, "mixer", "dim"), None, "dim"), (("layers", 1, "mixer", "heads"), 0, "heads"),
    (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"), (("layers", 0, "mixer", "scale"), None, "scale"),
    (("layers", 0, "mixer", "rot", "dims"), 18, "rot.dims"), (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 0, "mixer", "rot", "dims"), None, "rot.dims"), (("layers", 0, "mixer", "rot", "scaling", "low"), None, "scaling.low"),
    (("layers", 0, "mixer", "rot", "scaling", "low"), 5.0, "scaling.low"), (("layers", 0, "mixer", "rot", "scaling", "factor"), 0, "factor"),
    (("layers", 2, "mixer", "rot"), None, "rot"), (("layers", 2, "mixer", "q_rank"), 0, "q_rank"), (("layers", 2, "mixer", "kv_rank"), 1.5, "kv_rank"),
    (("layers", 2, "mixer", "rot", "dims"), 10, "rot.dims"), (("layers", 2, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mlp", "kind"), "dense", "mlp.kind"), (("layers", 0, "mlp", "router", "top"), 9, "router.top"),
    (("layers", 0, "mlp", "router", "identity"), -1, "router.identity"), (("layers", 0, "mlp", "expert"), None, "expert"),
    (("layers", 0, "mlp", "expert", "ff"), None, "ff"),
])
def test_errors_name_the_key(path, value, word):
    d = _cfg("fv_a")
    node = d
    for k in path[:-1]:
        node = node[k]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    with pytest.raises(PhotonError) as e:
        FezavikConfig.from_dict(d)
    assert e.value.code == ErrorCode.INVALID_CONFIG and word in str(e.value)


def test_parts_and_their_parameters():
    spec = load_spec("fv_a")
    a, r, c, b = spec.layers
    assert [l.block.kind for l in spec.layers] == ["sandwich"] * 4
    p = a.mixer.params
    assert a.mixer.kind == "normed_attention"
    assert (p["n_q_heads"], p["n_kv_heads"], p["head_dim"], p["value_dim"], p["scale"], p["window"], p["rot_dims"], p["rot_base"], p["rot_interleaved"],
            p["norm_weight"], p["norm_scope"], p["sink"]) == (6, 2, 16, 32, 0.3, 40, 8, 5000.0, True, True, "row", "learned")
    assert p["rot_scaling"] == {"factor": 4.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0, "original_max_position_embeddings": 64.0}
    assert b.mixer.params["rot_scaling"] is None
    assert r.mixer.kind == "hgrn2" and {k: r.mixer.params[k] for k in ("heads", "dim", "vdim", "eps")} == dict(heads=2, dim=12, vdim=20, eps=1e-5)
    p = c.mixer.params
    assert c.mixer.kind == "latent_attention"
    assert (p["heads"], p["dim"], p["rot_dim"], p["vdim"], p["kv_rank"], p["q_rank"], p["window"], p["rot_dims"], p["rot_base"], p["output_gate"],
            p["sink"], p.get("rot_interleaved", False)) == (3, 16, 8, 20, 24, 40, 17, 8, 500.0, "head", True, False)
    f = a.feed_forward.params
    assert (f["experts"], f["identity"], f["top"], f["expert_size"], f["scoring"], f["correction"], f["router_bias"], f["activation"]) == \
        (6, 2, 2, 32, "softmax_raw", True, False, "silu")
    assert [x.params["weight_name"] for x in (a.norm1, a.post1, a.norm2, a.post2)] == ["norm1", "norm1b", "norm2", "norm2b"]
    assert c.feed_forward is None and c.norm2 is None and c.post2 is None and c.post1 is not None
    assert spec.head_name == "head" and spec.embedding_scale is None
    assert load_spec("fv_e").layers[0].feed_forward.params["identity"] == 0 and load_spec("fv_b").layers[3].mixer.params["rot_dims"] == 20


def test_what_the_file_leaves_out_does_not_exist():
    p = load_spec("fv_e").layers[0].mixer.params
    assert p["window"] is None and p["rot_dims"] == 0 and p["rot_scaling"] is None
    d = _cfg("fv_a")
    d["layers"][0]["mixer"].pop("kv_heads"); d["layers"][0]["mixer"].pop("vdim")
    p = load_spec(d).layers[0].mixer.params
    assert p["n_kv_heads"] == 6 and p["value_dim"] == 16


def test_declared_tensors():
    d = declared_tensors(load_spec("fv_a"))
    for n in ("embed", "head", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.q", "l0.mix.k", "l0.mix.v", "l0.mix.q.norm",
              "l0.mix.k.norm", "l0.mix.sink", "l0.mix.o", "l0.mlp.router", "l0.mlp.correction", "l0.mlp.e5.gate", "l0.mlp.e0.up", "l0.mlp.e3.down",
              "l1.mix.q", "l1.mix.f", "l1.mix.f.b", "l1.mix.lower", "l1.mix.v", "l1.mix.norm", "l1.mix.o", "l2.mix.dq", "l2.mix.dq.norm",
              "l2.mix.uq", "l2.mix.dkv", "l2.mix.dkv.norm", "l2.mix.uk", "l2.mix.uv", "l2.mix.sink", "l2.mix.g", "l2.mix.o", "l2.norm1b"):
        assert n in d, n
    for n in ("l2.norm2", "l2.norm2b", "l0.mlp.e6.up", "l0.mlp.router.b", "l1.mix.k", "l1.mix.g", "l0.mix.g"):
        assert n not in d, n
    assert d["l0.mix.q.norm"].shape == (96,) and d["l0.mix.k.norm"].shape == (32,) and d["l0.mix.v"].shape == (64, 64) and d["l0.mix.o"].shape == (64, 192)
    assert d["l0.mlp.router"].shape == (8, 64) and d["l0.mlp.correction"].shape == (8,) and d["l0.mix.sink"].shape == (6,)
    assert d["l1.mix.f"].shape == (24, 64) and d["l1.mix.lower"].shape == (24,) and d["l1.mix.norm"].shape == (20,)
    assert d["l2.mix.g"].shape == (3, 64) and d["l2.mix.dkv"].shape == (32, 64)


def test_cache_needs():
    spec = load_spec("fv_a")
    sk = _Skeleton(spec)
    needs = [(sk.blocks[e.layer].mixer().cache_spec(), sk.blocks[e.layer].mixer().state_spec()) for e in spec.run]
    assert needs[0][0] == PagedCacheSpec(2, 16, 40, value_dim=32) and needs[3][0] == PagedCacheSpec(3, 32, 9, value_dim=16)
    assert needs[2][0] == PagedCacheSpec(1, 32, 17, values=False) and needs[1][0] is None
    assert needs[1][1].shape == (2 * 12 * 20,) and needs[1][1].dtype == torch.float32 and needs[0][1] is None
    cm = CacheManager(needs, [None] * 4, 8, 40, 2, torch.bfloat16, None)
    cm.add_request("r")
    cm.extend("r", 100)
    cm.commit("r", 100)
    for g in cm.groups:
        window = g.spec.window
        held = [i for i, p in enumerate(g.tables["r"]) if p >= 0]
        assert held[0] == (100 - window + 1) // 8 and held[-1] == 99 // 8


def test_a_file_may_carry_the_unused_norms_of_a_layer_without_feed_forward():
    assert load_spec("fv_a").ignored_tensors == ("l2.norm2", "l2.norm2b") and load_spec("fv_d").ignored_tensors == ("l2.norm2", "l2.norm2b")


@pytest.mark.parametrize("scaling", [None, (8.0, 1.0, 4.0, 512.0), (3.0, 0.5, 0.75, 40.0), (1.0, 1.0, 2.0, 64.0)])
@pytest.mark.parametrize("dims,base", [(2, 10.0), (32, 10000.0), (6, 777.0), (64, 3e5)])
def test_stretched_frequencies(scaling, dims, base):
    keys = ("factor", "low", "high", "original")
    long_keys = ("factor", "low_freq_factor", "high_freq_factor", "original_max_position_embeddings")
    want = plain.frequencies(dims, base, None if scaling is None else dict(zip(keys, scaling)))
    got = scaled_frequencies(dims, base, None if scaling is None else dict(zip(long_keys, scaling)))
    assert got.dtype == torch.float64 and torch.allclose(got, torch.tensor(want, dtype=torch.float64), rtol=1e-14)


def test_the_block_between_two_norms_in_plain_operations():
    """Norms without a fused kernel: the pending output passes its norm before the sum."""
    class Rms(Norm):
        def __init__(self, w, eps):
            self.w, self.eps = w, eps

        def forward(self, x, out_dtype):
            return plain.rms_norm(x.double(), self.w, self.eps).to(out_dtype)

    class Mix(Mixer):
        def forward(self, h, ctx, cache):
            return h.flip(-1) * 2

    class Ff(FeedForward):
        def forward(self, h, ctx):
            return torch.tanh(h)

    class Ctx:
        dtype = torch.float32
    g = torch.Generator().manual_seed(4)
    w = [1 + 0.3 * torch.randn(6, generator=g).double() for _ in range(4)]
    x = torch.randn(5, 6, generator=g)
    want = plain.sandwich(x.double(), lambda h: h.flip(-1) * 2, w[0], w[1], 1e-3)
    short = want
    want = plain.sandwich(want, torch.tanh, w[2], w[3], 1e-3)
    n = [Rms(v, 1e-3) for v in w]
    res, delta = SandwichBlock(n[0], Mix(), n[1], n[2], Ff(), n[3]).forward(x.clone(), None, Ctx, None)
    assert isinstance(delta, Normed) and torch.allclose((res + delta.materialize()).double(), want, atol=1e-5)
    res, delta = SandwichBlock(n[0], Mix(), n[1]).forward(x.clone(), None, Ctx, None)
    assert torch.allclose((res + delta.materialize()).double(), short, atol=1e-5)
    with pytest.raises(ValueError):
        SandwichBlock(n[0], Mix(), n[1], n[2])


def test_what_does_not_combine():
    base = dict(hidden_size=16, experts=2, top=1, expert_size=8)
    for bad in (dict(identity=2), dict(correction=True), dict(scoring="softmax_raw", groups=2), dict(scoring="softmax_raw", identity=1, top=4),
                dict(scoring="softmax_raw", identity=1, weight_input=True)):
        with pytest.raises(ValueError):
            create_part("feed_forward", "moe", dict(base, **bad))
    create_part("feed_forward", "moe", dict(base, scoring="softmax_raw", identity=1, top=3))
    with pytest.raises(ValueError):
        create_part("mixer", "normed_attention", dict(hidden_size=16, n_q_heads=2, n_kv_heads=1, head_dim=8, eps=1e-5, norm_scope="layer"))
    with pytest.raises(ValueError):
        create_part("mixer", "latent_attention", dict(hidden_size=16, heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=8, q_rank=8, scale=1.0, eps=1e-5,
                                                      rot_base=10.0, output_gate="row"))


def test_random_lower_bounds_lie_below_one(tmp_path):
    _, tensors = plain.read_folder(make_fezavik_folder(str(tmp_path / "m"), "fv_d"))
    low = tensors["l0.mix.lower"].float()
    assert float(low.min()) >= 0.0 and float(low.max()) < 1.0 and float(low.std()) > 0.15

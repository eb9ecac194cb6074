"""The Milozen configuration, its model spec, the tensors it declares, what the cache manager is asked for (one latent row
per token in the layers that own one, kept for the longest window among their readers), and the plain form of the
parallel residual streams; no GPU."""
import copy

import pytest
import torch

from helpers import TINY_MILOZEN, make_milozen_folder
from plain import milozen_plain as plain
from photon_infer_b200.cache.manager import CacheManager
from photon_infer_b200.config import load_config
from photon_infer_b200.config.milozen_config import MilozenConfig
from photon_infer_b200.errors import ErrorCode, PhotonError
from photon_infer_b200.models.model import _Skeleton, declared_tensors
from photon_infer_b200.parts.base import Connected, Norm, PagedCacheSpec, delta_pair
from photon_infer_b200.parts.registry import create_part


def _cfg(name):
    return copy.deepcopy(TINY_MILOZEN[name]["config"])


def load_spec(name_or_dict):
    from photon_infer_b200.config import get_architecture
    arch = get_architecture("Milozen")
    d = _cfg(name_or_dict) if isinstance(name_or_dict, str) else name_or_dict
    return arch.build_spec(arch.config_class.from_dict(d))


def test_round_trip_and_registry(tmp_path):
    for name in TINY_MILOZEN:
        cfg = MilozenConfig.from_dict(_cfg(name))
        assert MilozenConfig.from_dict(cfg.to_dict()) == cfg
    folder = make_milozen_folder(str(tmp_path / "m"), "mz_a")
    arch, cfg = load_config(folder)
    assert arch.name == "Milozen" and cfg.width == 64 and cfg.streams == 2 and cfg.embedding_scale == 4.0
    d = _cfg("mz_b"); d["architectures"] = [d.pop("architecture")]
    assert MilozenConfig.from_dict(d).architecture == "Milozen"


@pytest.mark.parametrize("path,value,word", [
    (("width",), None, "width"), (("vocab",), 0, "vocab"), (("streams",), None, "streams"), (("streams",), 0, "streams"),
    (("norm", "eps"), None, "norm.eps"), (("norm",), None, "norm"), (("embedding", "scale"), "x", "embedding.scale"),
    (("layers", 1, "type"), "attention", "layers[1].type"), (("layers", 0, "mixer", "dim"), None, "dim"),
    (("layers", 0, "mixer", "q_rank"), 0, "q_rank"), (("layers", 0, "mixer", "kv_rank"), 1.5, "kv_rank"),
    (("layers", 0, "mixer", "scale"), None, "scale"), (("layers", 0, "mixer", "rot"), None, "rot"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"), (("layers", 0, "mixer", "rot", "dims"), 10, "rot.dims"),
    (("layers", 0, "mixer", "rot", "base"), None, "rot.base"), (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 2, "mixer", "kv_from"), 2, "kv_from"), (("layers", 3, "mixer", "kv_from"), 2, "kv_from"),
    (("layers", 2, "mixer", "kv_from"), 1, "kv_rank"), (("layers", 2, "mixer", "rot", "base"), 10.0, "rot"),
    (("layers", 1, "mlp", "kind"), "glu", "mlp.kind"), (("layers", 1, "mlp", "ff"), None, "ff"),
    (("layers", 0, "mlp", "router", "top"), 9, "router.top"), (("layers", 0, "mlp", "expert", "limit"), None, "limit"),
    (("layers", 0, "mlp", "expert", "limit"), -1.0, "limit"), (("layers", 0, "mlp", "expert"), None, "expert"),
])
def test_errors_name_the_key(path, value, word):
    d = _cfg("mz_a")
    node = d
    for k in path[:-1]:
        node = node[k]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    with pytest.raises(PhotonError) as e:
        MilozenConfig.from_dict(d)
    assert e.value.code == ErrorCode.INVALID_CONFIG and word in str(e.value)


def test_parts_and_their_parameters():
    spec = load_spec("mz_a")
    a, b, reader, short = spec.layers
    assert [l.block.kind for l in spec.layers] == ["hyper_pre_norm"] * 4 and [l.mixer.kind for l in spec.layers] == ["latent_attention"] * 4
    p = a.mixer.params
    assert (p["heads"], p["dim"], p["rot_dim"], p["vdim"], p["kv_rank"], p["q_rank"], p["scale"], p["window"], p["rot_dims"],
            p["rot_base"], p["rot_interleaved"], p["own_kv"], p["output_gate"]) == (3, 16, 8, 20, 24, 40, 0.3, 40, 8, 5000.0, True, True, True)
    assert p["cache_window"] == 56 and b.mixer.params["cache_window"] == 17      # the longest reader's window; no reader
    assert reader.mixer.params["own_kv"] is False and reader.mixer.params["window"] == 56 and reader.mixer.params["heads"] == 5
    assert a.norm1.kind == "layer_norm" and a.norm1.params["bias_name"] is None and a.norm1.params["eps"] == 1e-5
    assert (a.connect1.kind, a.connect1.params, a.connect1.prefix, a.connect2.prefix) == ("hyper", {"streams": 2}, "hc1.", "hc2.")
    f = a.feed_forward.params
    assert a.feed_forward.kind == "moe" and (f["experts"], f["top"], f["expert_size"], f["scoring"], f["router_bias"], f["weight_input"],
                                             f["activation"], f["act_limit"], f["act_slope"]) == \
        (6, 2, 32, "sigmoid", False, True, "clamped_swish", 0.8, 1.702)
    assert b.feed_forward.kind == "gated" and b.feed_forward.params["activation"] == "silu"
    assert reader.feed_forward is None and reader.norm2 is None and reader.connect2 is None
    assert spec.head_name is None and spec.embedding_scale == 4.0                # the embedding table is the output head
    assert [(e.layer, e.kv_from) for e in spec.run] == [(0, None), (1, None), (2, 0), (3, 0)]
    e = load_spec("mz_e")                                                          # a reader without a window: all is kept
    assert e.layers[0].mixer.params["cache_window"] is None and e.layers[2].mixer.params["window"] == 8


def test_what_the_file_leaves_out_does_not_exist():
    d = _cfg("mz_a")
    d.pop("embedding")
    for l in d["layers"]:
        l["mixer"].pop("mask")
    spec = load_spec(d)
    assert spec.embedding_scale == 1.0
    assert all(l.mixer.params["window"] is None for l in spec.layers) and spec.layers[0].mixer.params["cache_window"] is None


def test_declared_tensors():
    d = declared_tensors(load_spec("mz_a"))
    for n in ("embed", "final.norm", "l0.norm1", "l0.norm2", "l0.hc1.in", "l0.hc1.out", "l0.hc1.mix", "l0.hc2.mix", "l0.mix.dq",
              "l0.mix.dq.norm", "l0.mix.uq", "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv", "l0.mix.g", "l0.mix.o",
              "l0.mlp.router", "l0.mlp.e5.gate", "l0.mlp.e0.up", "l0.mlp.e3.down", "l1.mlp.gate", "l1.mlp.up", "l1.mlp.down",
              "l2.mix.uk", "l2.mix.uv", "l2.hc1.mix"):
        assert n in d, n
    for n in ("head", "l2.mix.dkv", "l2.mix.dkv.norm", "l2.norm2", "l2.hc2.mix", "l0.norm1.b", "l0.mlp.router.b", "l0.mlp.e6.up"):
        assert n not in d, n
    assert d["l0.mix.uq"].shape == (3 * 24, 40) and d["l0.mix.dkv"].shape == (32, 64) and d["l0.mix.g"].shape == (60, 64)
    assert d["l2.mix.uk"].shape == (60, 24) and d["l2.mix.uv"].shape == (120, 24) and d["l2.mix.o"].shape == (64, 120)
    assert d["l0.hc1.mix"].shape == (2, 2) and d["l0.hc1.in"].shape == (2,)


def test_cache_needs_and_the_longest_reader_s_window():
    spec = load_spec("mz_a")
    sk = _Skeleton(spec)
    needs = [(sk.blocks[e.layer].mixer().cache_spec() if e.kv_from is None else None, None) for e in spec.run]
    assert needs[0][0] == PagedCacheSpec(1, 32, 56, values=False) and needs[1][0] == PagedCacheSpec(1, 48, 17, values=False)
    assert needs[2][0] is None and needs[3][0] is None
    cm = CacheManager(needs, [e.kv_from for e in spec.run], 8, 40, 2, torch.bfloat16, None)
    assert [g.entries for g in cm.groups] == [[0], [1]] and cm.entry_location[3] == cm.entry_location[0] and cm.entry_shared[2]
    cm.add_request("r")
    cm.extend("r", 100)
    cm.commit("r", 100)
    for g, window in ((0, 56), (1, 17)):
        held = [i for i, p in enumerate(cm.groups[g].tables["r"]) if p >= 0]
        assert held[0] == (100 - window + 1) // 8 and held[-1] == 99 // 8


def test_streams_written_and_read_by_plain_operations():
    """``Connected.apply`` and the default ``Norm.read_streams`` (what a norm without a kernel for streams uses), from
    streams that are all equal and from different ones."""
    class Twice(Norm):
        def forward(self, x, out_dtype):
            return (2 * x).to(out_dtype)

    g = torch.Generator().manual_seed(1)
    S, T, H = 3, 5, 7
    c = create_part("connection", "hyper", {"streams": S})
    w = {"in": torch.randn(S, generator=g), "out": torch.randn(S, generator=g), "mix": torch.randn(S, S, generator=g)}
    c.load(w)
    y, x0 = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g)
    X = torch.randn(T, S, H, generator=g)
    for streams, old in ((x0, torch.stack([x0] * S)), (X, X.transpose(0, 1))):
        want = plain.streams_write(old.double(), w["mix"].double(), w["out"].double(), y.double())
        new = Connected(y, c).apply(streams)
        assert torch.allclose(new.transpose(0, 1).double(), want, atol=1e-5)
        h, kept = Twice().read_streams(Connected(y, c), streams, c.w_in, torch.float32)
        assert torch.allclose(kept, new) and torch.allclose(h.double(), 2 * plain.streams_read(want, w["in"].double()), atol=1e-5)
        rows = torch.tensor([3, 0], dtype=torch.int32)
        last, same = Twice().read_streams(Connected(y, c), streams, None, torch.float32, rows)
        assert same is streams and torch.allclose(last.double(), 2 * want.sum(0)[[3, 0]], atol=1e-5)
        h0, _ = Twice().read_streams(None, streams, c.w_in, torch.float32)
        assert torch.allclose(h0.double(), 2 * plain.streams_read(old.double(), w["in"].double()), atol=1e-5)
    with pytest.raises(TypeError):
        delta_pair(Connected(y, c))
    with pytest.raises(ValueError):
        create_part("connection", "hyper", {"streams": 17})


def test_a_file_may_carry_the_unused_tensors_of_a_layer_without_feed_forward():
    assert load_spec("mz_a").ignored_tensors == ("l2.norm2", "l2.hc2.*")
    assert load_spec("mz_b").ignored_tensors == ()


def test_random_mix_matrices_are_near_the_identity(tmp_path):
    _, tensors = plain.read_folder(make_milozen_folder(str(tmp_path / "m"), "mz_b"))
    m = tensors["l0.hc1.mix"].float()
    assert float((m - torch.eye(4)).abs().max()) < 0.6 and float(m.diagonal().mean()) > 0.5

"""The Lilovik decoder: its name in config.json and the names of its tensors.

Layer i's tensors start with "l<i>."; a mixer's are "l<i>.mix.*", a feed-forward's "l<i>.mlp.*", the norms before and
after the mixer "l<i>.norm1" and "l<i>.norm1b", before and after the feed-forward "l<i>.norm2" and "l<i>.norm2b". The
frame's are "embed", "final.norm" and "head".
"""
from ..config.lilovik import LilovikConfig
from ..config.registry import register_architecture
from .layout import ModelLayout
from .model import expected_tensors

_ATTENTION = {"wq": "q", "wk": "k", "wv": "v", "bq": "q.b", "bk": "k.b", "bv": "v.b", "q_norm": "q.norm", "k_norm": "k.norm",
              "shift": "pb", "mix": "talk", "wo": "o"}
_AVERAGE = {"wz": "z", "bz": "z.b", "wu": "x", "bu": "x.b", "wg": "g", "wo": "o"}
_BY_KIND = {"attention": _ATTENTION, "gated_average": _AVERAGE}


class LilovikArchitecture:
    name = "Lilovik"

    def parse_config(self, raw):
        return LilovikConfig.from_dict(raw)

    def layout(self, spec):
        layers = []
        for l, block in enumerate(spec.layers):
            p = f"l{l}."
            names = {("mixer_norm", "weight"): p + "norm1", ("mixer_post_norm", "weight"): p + "norm1b"}
            for slot, short in _BY_KIND[block.mixer.kind].items():
                names[("mixer", slot)] = p + "mix." + short
            if block.ffn is not None:
                names.update({("ffn_norm", "weight"): p + "norm2", ("ffn_post_norm", "weight"): p + "norm2b"})
                for slot in ("gate", "up", "down"):
                    names[("ffn", slot)] = p + "mlp." + slot
            layers.append(names)
        return ModelLayout(embed="embed", final_norm="final.norm", head="head", layers=layers)

    def random_moments(self, name, shape, std, norm_std):
        """(mean, amplitude) of a random tensor of this design where the general rule (matrices around zero, vectors
        around one) does not fit; None: the general rule."""
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm1b", "norm2", "norm2b") or name == "final.norm":  # stored around zero
            return 0.0, norm_std
        if last == "b":
            return (-2.0 if name.endswith(".z.b") else 0.0), 0.5
        if last == "pb":
            return -3.0, 0.5
        return None

    def info(self, spec):
        kinds = "".join("a" if b.mixer.kind == "attention" else "r" for b in spec.layers)
        ffs = "".join("-" if b.ffn is None else "d" for b in spec.layers)
        return f"lilovik dim={spec.hidden} layers={len(spec.layers)} ({kinds}; feed-forwards {ffs}) vocab={spec.vocab}"

    def tensor_names(self, spec, available=None):
        return expected_tensors(spec, self.layout(spec), available)


register_architecture(LilovikArchitecture())

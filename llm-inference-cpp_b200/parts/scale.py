"""Parts of the family ``scale``: a learned factor per entry on what a sublayer adds to the stream.  The arrangement hands the
vector to the sublayer (``out_scale=``), whose last product multiplies by it before it adds."""
from __future__ import annotations

from .registry import TensorDecl, part


@part("scale", "vector")
class ScaleVector:
    """params: ``width``.  tensors (the prefix is the tensor's full name): ``""`` [width], kept in fp32 as ``weight``."""
    takes_padding_rows = True       # rows are treated alone

    @classmethod
    def declare(cls, spec):
        return {"": TensorDecl((spec.params["width"],), "norm_scale")}

    def __init__(self, spec, tensors, rt, **_):
        self.weight = rt.to_f32(tensors[""]).contiguous()

"""Step engine of Mopalorn: the shared packed-batch engine with the family's step function."""
from ..step_engine import StepEngine
from . import model


class MopalornEngine(StepEngine):
    make_cache = staticmethod(model.make_cache)
    make_rope = staticmethod(model.make_rope)
    run_layers = staticmethod(model.run_layers)
    output_logits = staticmethod(model.output_logits)

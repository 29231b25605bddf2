from .modeling_dekutar import (  # noqa: F401
    DekutarConfig, DekutarModel, DekutarForCausalLM, DekutarForSequenceClassification, DekutarLayerPolicy, DekutarBlock,
    DekutarPreTrainedModel)
